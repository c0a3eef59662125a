"""Host side of the Subivik family: registry, files, shared keys, state and cache sizes, configuration checks."""
import json

import pytest
import torch
import torch.nn.functional as F

from minivllm_b200.engine import cache
from minivllm_b200.engine.registry import build_model, family_of, folder_config
from minivllm_b200.engine.subivik import SubivikConfig, SubivikForCausalLM
from minivllm_b200.engine.weights import DictWeights, RandomWeights
from minivllm_b200.layers.tanh_norm import position_frequencies
from minivllm_b200.layers.window_attention import chunk_keys, window_keys
from minivllm_b200.utils.context import Context
from oracle import subivik_oracle as oracle
from tests import subivik_cases as cases
from tests.test_sipazen_host import _write


def _build(cfg, w):
    return SubivikForCausalLM(SubivikConfig.from_dict(cfg), dtype=torch.float32, device="cpu",
                              weights=DictWeights(w, torch.float32, "cpu"))


def test_family_is_chosen_by_architecture(tmp_path):
    cfg, w = cases.model("odd")
    assert family_of(cfg).model is SubivikForCausalLM
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    _write(tmp_path / "model.safetensors", w)
    c = folder_config(str(tmp_path), block_size=32)
    m = build_model(c, SubivikConfig.from_dict(c), 0, 1, torch.float32, "cpu")
    assert torch.equal(m.layers[1].mixer.left.talk, w["l1.mix.left.talk"].float())
    assert m.lm_head is m.embed and m.layers[0].mixer.scale == 19 ** -0.5
    assert m.layers[3].mixer.scales == (1.3, 0.7) and m.layers[1].entry1.alpha == float(w["l1.norm1.alpha"])


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_tensor_is_used(name):
    cfg, w = cases.model(name)
    m = _build(cfg, w)
    assert [l.mlp is None for l in m.layers] == [l["mlp"] is None for l in cfg["layers"]]
    with pytest.raises(ValueError, match="belong to no part"):
        _build(cfg, {**w, "l0.mix.extra": torch.zeros(1)})
    for missing in ("l0.norm1.b", "l0.norm1.alpha", "l1.norm1", "final.norm.b", "embed"):
        with pytest.raises((KeyError, ValueError)):
            _build(cfg, {k: v for k, v in w.items() if k != missing})
    seeded = SubivikForCausalLM(SubivikConfig.from_dict(cfg), dtype=torch.float32, device="cpu",
                                weights=RandomWeights(1, torch.float32, "cpu"))
    assert seeded.cfg.widest_activation() > 0 and len(seeded.layers) == len(cfg["layers"])


def test_cache_and_state_sizes():
    """Layers that use another's keys have no cache rows of their own; time mixing keeps its matrix and the last input."""
    cfg, w = cases.model("odd")
    m = _build(cfg, w)
    row, state = 0, 0
    for l in cfg["layers"]:
        s = l["mixer"]
        if l["type"] == "parallel":
            a, b = s["left"], s["right"]
            row += a["kv_heads"] * (a["dim"] + a["vdim"])
            state += 4 * b["heads"] * b["dim"] ** 2 + 2 * cfg["width"]
        elif "kv_from" not in s:
            row += s["kv_heads"] * (2 * s["dim"] + s["vdim"])
    assert cache.paged_block_bytes(m, 16, torch.bfloat16) == row * 32 and len(cache.paged_modules(m)) == 3
    assert cache.slot_bytes(m, torch.bfloat16) == state
    cache.bind(m, 3, 16, 2, torch.float32, "cpu")
    assert m.layers[2].mixer._source[0].paged_cache is m.layers[0].mixer.paged_cache and m.layers[0].mixer.lends
    assert not cache.state_modules(_build(*cases.model("attention_only")))


def test_constants_of_a_layer():
    cfg, w = cases.model("odd")
    m = _build(cfg, w)
    d = {k: t.double() for k, t in w.items()}
    want = oracle.difference_factor(*(d["l2.mix." + n] for n in ("lq1", "lk1", "lq2", "lk2")), 0.3)
    assert abs(m.layers[2].mixer.lam - float(want)) < 1e-6 and m.layers[2].mixer.mult == 1 - 0.3
    p, q = (oracle.softplus(x) for x in d["l4.mlp.act"])
    assert abs(m.layers[4].mlp.a - float(p)) < 1e-6 and abs(m.layers[4].mlp.b - 0.5 - float(q)) < 1e-6
    assert m.layers[0].mlp.scale == 1.7 and m.layers[0].mlp.over_all
    f = position_frequencies(7, "cpu")
    assert f.dtype == torch.float64 and f.numel() == 4 and float(f[3]) == 10000.0 ** (-6 / 7)


def test_output_product_joins_both_mixers():
    cfg, w = cases.model("odd")
    mixer = _build(cfg, w).layers[1].mixer
    assert mixer.at == 60 and mixer.o_w.shape == (91, 60 + 33)
    a, b = torch.randn(4, 60), torch.randn(4, 33)
    torch.testing.assert_close(F.linear(torch.cat([a, b], 1), mixer.o_w),
                               a @ w["l1.mix.left.o"].float().T + b @ w["l1.mix.right.o"].float().T, rtol=1e-4, atol=1e-4)
    assert mixer.shift is mixer.right.shift and mixer.right.shift.mu.shape == (5, 91)
    rank = w["l1.mix.right.w1"].shape[0]         # padded to whole 16-byte pieces without a change of the product
    assert mixer.right.w1_w.shape == (8, 91) and bool((mixer.right.w1_w[rank:] == 0).all()) and bool((mixer.right.w2_w[:, rank:] == 0).all())


def test_keys_that_portions_see(monkeypatch):
    monkeypatch.setattr(torch.Tensor, "pin_memory", lambda t: t)
    ctx = Context(portion_spans=[(0, 5), (119, 2), (120, 7), (250, 30)])
    cu, first, total = chunk_keys(ctx, 120, "cpu")
    assert first.tolist() == [0, 0, 120, 240] and cu.tolist() == [0, 5, 126, 133, 173] and total == 173
    cu, first, total = window_keys(ctx, 120, "cpu")
    assert first.tolist() == [0, 0, 1, 131] and total == 5 + 121 + 126 + 149
    assert chunk_keys(ctx, 1, "cpu")[1].tolist() == [0, 119, 120, 250]


def test_configuration_errors():
    cfg, w = cases.model("odd")
    def changed(f):
        c = json.loads(json.dumps(cfg))
        f(c)
        return c
    bad = {"unknown mixer": lambda c: c["layers"][0].update(type="nothing"),
           "unknown feed-forward": lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
           "kv_from": lambda c: c["layers"][2]["mixer"].update(kv_from=1),
           "kv_from 4": lambda c: c["layers"][4]["mixer"].update(kv_from=4)}
    for text, f in bad.items():
        with pytest.raises(ValueError, match=text.split()[0]):
            SubivikConfig.from_dict(changed(f))
    for f in (lambda c: c["layers"][4]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(vdim=7),
              lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), lambda c: c["layers"][1]["mixer"]["left"].update(softcap=0.0),
              lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4)):
        with pytest.raises(ValueError):
            _build(changed(f), w)
    with pytest.raises(ValueError, match="one GPU"):
        SubivikForCausalLM(SubivikConfig.from_dict(cfg), tp_size=2)
    with pytest.raises(ValueError, match="float32"):
        SubivikForCausalLM(SubivikConfig.from_dict(cfg), dtype=torch.float16)


def test_oracle_mechanisms():
    """The oracle's pieces against facts that need no second implementation."""
    eye = torch.eye(3, dtype=torch.float64)
    q, k, v = (torch.randn(9, n, 4, dtype=torch.float64) for n in (6, 3, 3))
    one = torch.zeros(6, dtype=torch.float64)
    w = oracle.capped_weights(q, k, one, one, 0.5, 1e9)
    plain = torch.softmax((torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(2, 1)) * 0.5).masked_fill(~torch.ones(9, 9).tril().bool(), -1e30), -1)
    torch.testing.assert_close(w, plain)
    assert torch.equal(oracle.mix_heads(w[:3], eye), w[:3])
    a = oracle.chunk_attention(q, k, v, 0.5, 4)
    torch.testing.assert_close(a[4:8], oracle.chunk_attention(q[4:8], k[4:8], v[4:8], 0.5, 4))
    o, S = oracle.bonus_scan(q, q, q, torch.ones_like(q), torch.ones(6, 4, dtype=torch.float64))
    torch.testing.assert_close(o, torch.einsum("ihk,jhk,jhv,ij->ihv", q, q, q, torch.ones(9, 9, dtype=torch.float64).tril()))
    idx, weight = oracle.route(torch.randn(5, 7, dtype=torch.float64), 7, 2.0)
    torch.testing.assert_close(weight.sum(-1), torch.full((5,), 2.0, dtype=torch.float64))
    z = torch.tensor([-1e-9, 1e-9, -30.0, 2.0], dtype=torch.float64)
    p = torch.tensor(0.3, dtype=torch.float64)
    got = oracle.xielu(z, p, p)
    sp = float(oracle.softplus(p))
    torch.testing.assert_close(got, torch.tensor([-5e-10, 5e-10, (0.5 + sp) * 29.0 - 15.0, 4 * sp + 1.0], dtype=torch.float64))
