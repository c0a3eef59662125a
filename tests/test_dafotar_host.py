"""Host side of the Dafotar family: registry, files, weight order, shared keys, configuration checks."""
import json

import pytest
import torch

from minivllm_b200.engine import cache
from minivllm_b200.engine.dafotar import DafotarConfig, DafotarForCausalLM
from minivllm_b200.engine.registry import build_model, family_of, folder_config
from minivllm_b200.engine.weights import DictWeights, RandomWeights
from minivllm_b200.layers import rotary_attention as RA
from tests import dafotar_cases as cases
from tests.test_sipazen_host import _write


def _build(cfg, w):
    return DafotarForCausalLM(DafotarConfig.from_dict(cfg), dtype=torch.float32, device="cpu",
                              weights=DictWeights(w, torch.float32, "cpu"))


def test_family_is_chosen_by_architecture(tmp_path):
    cfg, w = cases.model("odd")
    assert family_of(cfg).model is DafotarForCausalLM
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    _write(tmp_path / "model.safetensors", w)
    c = folder_config(str(tmp_path), block_size=32)
    m = build_model(c, DafotarConfig.from_dict(c), 0, 1, torch.float32, "cpu")
    assert torch.equal(m.layers[2].mixer.temp, w["l2.mix.temp"].float())
    assert m.lm_head is m.embed and m.layers[0].mixer.scale == 19 ** -0.5


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_tensor_is_used(name):
    cfg, w = cases.model(name)
    m = _build(cfg, w)
    assert [l.mlp is None for l in m.layers] == [l["mlp"] is None for l in cfg["layers"]]
    with pytest.raises(ValueError, match="belong to no part"):
        _build(cfg, {**w, "l0.mix.extra": torch.zeros(1)})
    for missing in ("l0.norm1.b", "l0.hc1.mix", "l0.canon1", "final.norm.b"):
        with pytest.raises((KeyError, ValueError)):
            _build(cfg, {k: v for k, v in w.items() if k != missing})
    seeded = DafotarForCausalLM(DafotarConfig.from_dict(cfg), dtype=torch.float32, device="cpu",
                                weights=RandomWeights(1, torch.float32, "cpu"))
    assert seeded.cfg.widest_activation() > 0 and len(seeded.layers) == len(cfg["layers"])


def test_cache_and_state_sizes():
    """Layers that use another's keys have no cache rows of their own; every layer keeps its convolution's inputs."""
    cfg, w = cases.model("odd")
    m = _build(cfg, w)
    rows = [l["mixer"] for l in cfg["layers"] if l["type"] == "attention" and "kv_from" not in l["mixer"]]
    assert len(rows) == 1 and len(cache.paged_modules(m)) == 1
    assert cache.paged_block_bytes(m, 16, torch.bfloat16) == sum(r["kv_heads"] * (r["dim"] + r["vdim"]) for r in rows) * 32
    want = len(cfg["layers"]) * (cfg["canon"]["taps"] - 1) * cfg["width"] * 2
    for l in cfg["layers"]:
        s = l["mixer"]
        if l["type"] == "mlstm":
            want += 4 * s["heads"] * (s["dim"] * s["vdim"] + s["dim"] + 1)
    assert cache.slot_bytes(m, torch.bfloat16) == want
    cache.bind(m, 3, 16, 2, torch.float32, "cpu")
    assert m.layers[2].mixer._source[0].paged_cache is m.layers[0].mixer.paged_cache


def test_configuration_errors():
    cfg, w = cases.model("odd")
    def changed(f):
        c = json.loads(json.dumps(cfg))
        f(c)
        return c
    bad = {"unknown mixer": lambda c: c["layers"][0].update(type="nothing"),
           "unknown feed-forward": lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
           "kv_from": lambda c: c["layers"][2]["mixer"].update(kv_from=1),
           "kv_from 4": lambda c: c["layers"][4]["mixer"].update(kv_from=4),
           "streams": lambda c: c.update(streams=0)}
    for text, f in bad.items():
        with pytest.raises(ValueError, match=text.split()[0]):
            DafotarConfig.from_dict(changed(f))
    for f in (lambda c: c["layers"][4]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"]["rot"].update(base=7.0),
              lambda c: c["layers"][0]["mixer"]["rot"].update(dims=20), lambda c: c["layers"][1]["mixer"].update(gate_cap=0)):
        with pytest.raises(ValueError):
            _build(changed(f), w)
    with pytest.raises(ValueError, match="one GPU"):
        DafotarForCausalLM(DafotarConfig.from_dict(cfg), tp_size=2)
    with pytest.raises(ValueError, match="float32"):
        DafotarForCausalLM(DafotarConfig.from_dict(cfg), dtype=torch.float16)


def test_pairs_become_neighbours():
    assert RA.pair_order(7, 4) == [0, 2, 1, 3, 4, 5, 6] and RA.pair_order(6, 6) == [0, 3, 1, 4, 2, 5]
    assert RA.pair_order(5, 0) == list(range(5)) and RA.pair_order(2, 2) == [0, 1]
    w = torch.arange(24.0).view(12, 2)
    got = RA._reorder(w, 2, RA.pair_order(6, 4))
    for h in range(2):
        for i in range(2):
            assert torch.equal(got[6 * h + 2 * i], w[6 * h + i]) and torch.equal(got[6 * h + 2 * i + 1], w[6 * h + i + 2])
    assert torch.equal(RA._reorder(w.t(), 2, RA.pair_order(6, 4), dim=1), got.t())
    cfg, w = cases.model("odd")
    m = _build(cfg, w)
    x = torch.randn(5, 90, generator=torch.Generator().manual_seed(1))
    q = m.layers[0].mixer.stacked(x)["q"].view(5, 6, 19)
    plain = (x @ w["l0.mix.q"].float().t()).view(5, 6, 19)
    torch.testing.assert_close(q, plain[..., RA.pair_order(19, 12)])
