"""Small Fozerax configurations and helpers shared by the tests."""
import functools

import torch

from oracle import fozerax_oracle as oracle
from tests.sipazen_cases import check, error  # noqa: F401  (re-exported)


def _gla(heads, dim, vdim, tau):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def _par(heads, kv, dim, vdim, window, bias_max, right, scale=None):
    rh, rkv, rdim, rvdim, conv = right
    return "parallel", {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "bias_max": bias_max, "mask": {"size": window},
                 "scale": scale if scale is not None else dim ** -0.5},
        "right": {"heads": rh, "kv_heads": rkv, "dim": rdim, "vdim": rvdim, "conv": conv}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit, groups=None, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Fozerax", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


def odd():
    """No size is a multiple of eight, no two sizes agree; a layer without feed-forward, no shared expert."""
    return _config(131, 90, [
        (_gla(3, 14, 10, 5.0), _moe(9, 2, 22, 0.7, groups=(3, 2), shared=(34, 1.1))),
        (_par(6, 2, 18, 13, 11, 23, (6, 3, 10, 15, 3)), None),
        (_par(3, 3, 7, 9, 29, 64, (4, 1, 21, 6, 2), scale=0.4), _moe(5, 3, 19, 2.0)),
        (_gla(2, 37, 41, 2.5), _dense(46))], eps=1e-4)


def even():
    """Sizes that the tensor-core kernels take, windows shorter and longer than a tile of keys."""
    return _config(320, 192, [
        (_par(8, 2, 64, 128, 33, 100, (4, 2, 64, 128, 4)), _moe(8, 2, 128, 1.5, groups=(4, 3), shared=(64, 2.5))),
        (_gla(2, 128, 64, 16.0), _dense(256)),
        (_par(4, 1, 128, 64, 150, 90, (2, 2, 128, 128, 4)), _moe(6, 3, 64, 0.9)),
        (_gla(4, 32, 96, 8.0), _moe(8, 4, 72, 1.0, groups=(2, 1), shared=(192, 1.0)))])


def between():
    """Sizes that some of the tensor-core kernels take and others do not; wide heads."""
    return _config(257, 136, [
        (_par(3, 1, 40, 24, 57, 20, (3, 1, 72, 36, 5)), _dense(44)),
        (_gla(1, 200, 52, 3.0), None),
        (_par(4, 2, 136, 96, 24, 30, (2, 1, 130, 20, 2), scale=0.05), _moe(3, 2, 40, 1.2)),
        (_par(2, 2, 200, 160, 9, 40, (5, 5, 33, 8, 4), scale=0.05), _moe(4, 1, 16, 3.0, groups=(2, 2), shared=(20, 0.6)))])


def ones():
    """Sizes of one: a single head, tap, expert or key per window."""
    return _config(67, 40, [
        (_par(1, 1, 8, 16, 1, 12, (1, 1, 8, 24, 1)), _moe(1, 1, 24, 1.0)),
        (_gla(1, 8, 8, 1.0), _dense(8)),
        (_par(16, 1, 16, 8, 5, 9, (2, 1, 1, 3, 2)), _moe(2, 1, 8, 0.5, groups=(2, 1)))])


def gla_only():
    return _config(200, 64, [(_gla(2, 32, 32, 12.0), _dense(96))] * 2)


def parallel_only():
    return _config(200, 64, [(_par(4, 2, 32, 32, 20, 50, (2, 1, 32, 32, 4)), _moe(4, 2, 32, 1.0, shared=(32, 1.0)))] * 2)


CONFIGS = {"odd": odd, "even": even, "between": between, "ones": ones, "gla_only": gla_only, "parallel_only": parallel_only}


@functools.lru_cache(maxsize=None)
def model(name):
    cfg = CONFIGS[name]()
    return cfg, oracle.random_weights(cfg, seed=len(name), rank=3 + len(name), buckets=6 + 2 * len(name))


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
