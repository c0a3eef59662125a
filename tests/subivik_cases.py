"""Small Subivik configurations and helpers shared by the tests."""
import functools

import torch

from oracle import subivik_oracle as oracle
from tests.sipazen_cases import error


def _par(left, right, cap=18.0, scale=None, left_scale=0.9, right_scale=0.6):
    """left (heads, kv_heads, dim, vdim), right (heads, dim)."""
    H, G, d, vd = left
    return "parallel", {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": vd, "softcap": cap,
                                 "scale": scale if scale is not None else d ** -0.5},
                        "right": {"heads": right[0], "dim": right[1]}, "left_scale": left_scale, "right_scale": right_scale}


def _att(heads, kv, dim, vdim, chunk, diff=0.55, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "diff": diff,
         "scale": scale if scale is not None else dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def _moe(experts, top, ff, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Subivik", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": mlp} for (t, m), mlp in layers]}


def odd():
    """No size is a multiple of eight, no two sizes agree; every mixer with and without a feed-forward; layers that use an
    earlier one's keys through longer and shorter chunks."""
    return _config(131, 91, [
        (_att(6, 2, 19, 14, 11), _moe(7, 3, 21)),
        (_par((6, 3, 13, 10), (3, 11), cap=3.0), _dense(46)),
        (_att(6, 2, 19, 14, 37, diff=0.3, scale=0.4, kv_from=0), None),
        (_par((5, 1, 22, 9), (2, 37), cap=9.0, left_scale=1.3, right_scale=0.7), None),
        (_att(6, 2, 19, 14, 6, diff=0.75, kv_from=0), _dense(35))], eps=1e-4)


def even():
    """Sizes that the tensor-core kernels take, chunks shorter and longer than a tile of keys."""
    return _config(320, 192, [
        (_par((6, 3, 64, 128), (3, 64)), None),
        (_att(8, 2, 64, 128, 33), _dense(256)),
        (_par((6, 2, 128, 64), (1, 128), cap=30.0), _moe(16, 4, 40)),
        (_att(8, 2, 64, 128, 150, diff=0.4, kv_from=1), _moe(8, 2, 64, scale=2.5)),
        (_att(4, 4, 128, 64, 70), _dense(72))])


def between():
    """Sizes that some of the tensor-core kernels take and others do not; many heads over one, wide values."""
    return _config(257, 136, [
        (_par((20, 1, 40, 24), (2, 52)), _moe(5, 5, 24, scale=1.0)),
        (_att(9, 1, 72, 200, 57), None),
        (_par((3, 3, 136, 256), (1, 200), cap=50.0, scale=0.05), _dense(44)),
        (_att(2, 1, 160, 96, 24, scale=0.05), None),
        (_par((2, 1, 64, 192), (4, 24), cap=100.0), _dense(30))])


def ones():
    """Sizes of one: a single head, channel, expert, or key per chunk."""
    return _config(67, 40, [
        (_par((1, 1, 8, 16), (1, 8)), _dense(24)),
        (_att(1, 1, 8, 16, 1), _moe(1, 1, 8, scale=0.7)),
        (_par((4, 4, 1, 3), (1, 1), cap=2.0), None),
        (_att(16, 1, 16, 8, 5, diff=0.0), None)])


def parallel_only():
    return _config(200, 64, [(_par((2, 1, 32, 32), (2, 32)), _dense(96)), (_par((2, 2, 32, 48), (2, 32), cap=5.0), None)])


def attention_only():
    """No state: decoded tokens need the cache alone."""
    return _config(200, 64, [(_att(4, 2, 32, 32, 20), _dense(64)), (_att(4, 4, 32, 48, 1 << 20), None)])


CONFIGS = {f.__name__: f for f in (odd, even, between, ones, parallel_only, attention_only)}


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


# 32-bit: a few hundred roundings of 2^-24.  bfloat16: a hundred roundings of 2^-9.
LIMIT = {torch.float32: 1e-5, torch.bfloat16: 0.05}


def check(got, want, dtype):
    e = error(got, want)
    if dtype == torch.float32:
        assert float(e.max()) < LIMIT[dtype], f"worst {float(e.max()):.2e} at row {int(e.argmax())}"
    else:
        assert float(e.median()) < LIMIT[dtype] / 2, f"median {float(e.median()):.3f}"
        assert int((e > LIMIT[dtype]).sum()) <= max(1, e.numel() // 20), f"rows over the limit: {e[e > LIMIT[dtype]].tolist()}"
