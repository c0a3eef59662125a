"""Small Sipazen configurations and helpers shared by the tests."""
import functools

import torch

from oracle import sipazen_oracle as oracle


def _attention(heads, dim, rot, vdim, rank, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
            "scale": scale if scale is not None else (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}}


def _mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _moe(experts, top, ff, shared):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _config(vocab, width, groups, mult, layers, eps=1e-5):
    return {"architecture": "Sipazen", "vocab": vocab, "width": width, "residual_mult": mult,
            "norm": {"eps": eps, "groups": groups},
            "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers]}


def odd():
    """No size is a multiple of eight, no two sizes agree; a layer without feed-forward, experts of several kinds."""
    return _config(131, 90, 3, 0.45, [
        ("mamba2", _mamba(6, 10, 14, 3, 3, 2), _moe(5, 3, 22, 34)),
        ("latent_attention", _attention(3, 18, 6, 14, 26), None),
        ("latent_attention", _attention(5, 6, 10, 22, 38, base=500.0, scale=0.31), _moe(7, 1, 30, None)),
        ("mamba2", _mamba(4, 22, 9, 1, 2, 4), None)], eps=1e-4)


def even():
    """Sizes that the tensor-core kernels take."""
    return _config(320, 192, 4, 0.8, [
        ("latent_attention", _attention(4, 64, 32, 64, 128), _moe(8, 2, 128, 64)),
        ("mamba2", _mamba(8, 64, 64, 2, 4, 2), _moe(6, 3, 64, 192)),
        ("mamba2", _mamba(4, 64, 128, 1, 4, 1), _moe(4, 4, 72, 64)),
        ("latent_attention", _attention(16, 48, 64, 80, 256), _moe(8, 2, 64, 128))])


def between():
    """Sizes that some of the tensor-core kernels take and others do not."""
    return _config(257, 136, 2, 0.9, [
        ("latent_attention", _attention(3, 36, 28, 40, 68), _moe(9, 2, 44, 24)),
        ("mamba2", _mamba(3, 20, 32, 1, 4, 3), _moe(3, 2, 40, 136)),
        ("latent_attention", _attention(2, 36, 32, 24, 64, base=300.0), _moe(5, 2, 16, 20)),
        ("mamba2", _mamba(2, 56, 32, 2, 5, 7), _moe(3, 1, 48, None)),
        ("mamba2", _mamba(6, 24, 48, 3, 2, 1), _moe(6, 5, 8, 8))])


def attention_only():
    return _config(200, 64, 1, 1.0, [("latent_attention", _attention(2, 16, 16, 16, 32), _moe(4, 2, 32, 32))] * 2)


def mamba_only():
    return _config(200, 64, 2, 0.6, [("mamba2", _mamba(2, 32, 16, 1, 4, 1), _moe(4, 2, 32, 32))] * 2)


CONFIGS = {"odd": odd, "even": even, "between": between, "attention_only": attention_only, "mamba_only": mamba_only}


@functools.lru_cache(maxsize=None)
def model(name):
    cfg = CONFIGS[name]()
    w = oracle.random_weights(cfg, seed=len(name))
    if name == "between":
        # few experts and many layers: spread the router's logits, so that rounding does not swap the last expert chosen
        # with the first one that is not
        g = torch.Generator().manual_seed(1)
        for k in [k for k in w if k.endswith("mlp.router")]:
            w[k] = (w[k].float() * 0.3).to(torch.bfloat16)
            w[k + ".b"] = (1.5 * torch.randperm(w[k].shape[0], generator=g)).to(torch.bfloat16)
    return cfg, w


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


def error(got, want):
    """Per position: RMS of the difference of centred logits over the RMS of the centred logits."""
    want = want.double()
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    c = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / c.pow(2).mean().sqrt()


# 32-bit: a few hundred roundings of 2^-24.  bfloat16: a hundred roundings of 2^-9, and a router that now and then
# prefers another expert between two that are nearly tied.
LIMIT = {torch.float32: 2e-5, torch.bfloat16: 0.08}


def check(got, want, dtype):
    e = error(got, want)
    if dtype == torch.float32:
        assert float(e.max()) < LIMIT[dtype], f"worst {float(e.max()):.2e} at row {int(e.argmax())}"
    else:
        assert float(e.median()) < LIMIT[dtype] / 2, f"median {float(e.median()):.3f}"
        assert int((e > LIMIT[dtype]).sum()) <= max(1, e.numel() // 10), f"rows over the limit: {e[e > LIMIT[dtype]].tolist()}"
