"""Host side of the Fozerax family: registry, sizes that tensors fix by their shape, configuration checks."""
import json

import pytest
import torch

from minivllm_b200.engine import cache
from minivllm_b200.engine.fozerax import FozeraxConfig, FozeraxForCausalLM
from minivllm_b200.engine.registry import build_model, family_of, folder_config
from minivllm_b200.engine.weights import DictWeights, RandomWeights
from minivllm_b200.layers import window_attention as WA
from oracle import fozerax_oracle as oracle
from tests import fozerax_cases as cases
from tests.test_sipazen_host import _write


def _build(cfg, w):
    return FozeraxForCausalLM(FozeraxConfig.from_dict(cfg), dtype=torch.float32, device="cpu",
                              weights=DictWeights(w, torch.float32, "cpu"))


def test_family_is_chosen_by_architecture(tmp_path):
    cfg, w = cases.model("odd")
    assert family_of(cfg).model is FozeraxForCausalLM
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    _write(tmp_path / "model.safetensors", w)
    c = folder_config(str(tmp_path), block_size=32)
    m = build_model(c, FozeraxConfig.from_dict(c), 0, 1, torch.float32, "cpu")
    assert torch.equal(m.layers[1].mixer.left.sink, w["l1.mix.left.sink"].float())


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_every_tensor_is_used_and_sizes_come_from_tensors(name):
    cfg, w = cases.model(name)
    m = _build(cfg, w)
    for i, layer in enumerate(cfg["layers"]):
        mix = m.layers[i].mixer
        if layer["type"] == "gla":
            assert mix.a2_w.shape[1] == w[f"l{i}.mix.a1"].shape[0] != 16
        else:
            assert mix.left.bias.shape[0] == layer["mixer"]["left"]["heads"]
    with pytest.raises(ValueError, match="belong to no part"):
        _build(cfg, {**w, "l0.mix.extra": torch.zeros(1)})
    with pytest.raises((KeyError, ValueError)):
        _build(cfg, {k: v for k, v in w.items() if k != "l0.norm1"})
    seeded = FozeraxForCausalLM(FozeraxConfig.from_dict(cfg), dtype=torch.float32, device="cpu",
                                weights=RandomWeights(1, torch.float32, "cpu"))
    assert seeded.cfg.widest_activation() > 0 and len(seeded.layers) == len(cfg["layers"])


def test_cache_and_state_sizes():
    cfg, w = cases.model("odd")
    m = _build(cfg, w)
    rows = [l["mixer"]["left"] for l in cfg["layers"] if l["type"] == "parallel"]
    assert cache.paged_block_bytes(m, 16, torch.bfloat16) == sum(r["kv_heads"] * (r["dim"] + r["vdim"]) for r in rows) * 32
    want = 0
    for l in cfg["layers"]:
        s = l["mixer"] if l["type"] == "gla" else l["mixer"]["right"]
        want += 4 * s["heads"] * s["dim"] * s["vdim"]
        if l["type"] == "parallel":
            want += 2 * (s["conv"] - 1) * (2 * s["kv_heads"] * s["dim"] + s["heads"] * s["vdim"])
    assert cache.slot_bytes(m, torch.bfloat16) == want


def test_configuration_errors():
    cfg = cases.odd()
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "nothing"
    with pytest.raises(ValueError, match="unknown mixer"):
        FozeraxConfig.from_dict(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        FozeraxConfig.from_dict(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["router"]["groups"] = {"count": 3, "keep": 1}
    bad["layers"][0]["mlp"]["router"]["top"] = 4
    with pytest.raises(ValueError, match="moe"):
        _build(bad, cases.model("odd")[1])
    with pytest.raises(ValueError, match="one GPU"):
        FozeraxForCausalLM(FozeraxConfig.from_dict(cfg), tp_size=2)
    with pytest.raises(ValueError, match="float32"):
        FozeraxForCausalLM(FozeraxConfig.from_dict(cfg), dtype=torch.float16)


def test_distance_buckets():
    for buckets, bias_max in ((10, 23), (32, 128), (6, 4), (7, 40)):
        got = WA.distance_buckets(5 * bias_max, buckets, bias_max)
        assert got == [oracle.distance_bucket(n, buckets, bias_max) for n in range(5 * bias_max)]
        assert got[bias_max:] == [buckets - 1] * (4 * bias_max)
    with pytest.raises(ValueError):
        WA.distance_buckets(9, 8, 4)


def test_window_keys_of_a_step(monkeypatch):
    """Portions see the cached keys that their first query's window reaches, and their own."""
    from minivllm_b200.utils.context import Context
    monkeypatch.setattr(torch.Tensor, "pin_memory", lambda t: t)
    ctx = Context(portion_spans=[(0, 5), (3, 4), (100, 2), (20, 7)])
    cu, first, total = WA.window_keys(ctx, 21, "cpu")
    assert first.tolist() == [0, 0, 80, 0] and cu.tolist() == [0, 5, 12, 34, 61] and total == 61
    assert WA.window_keys(ctx, 21, "cpu")[0] is not None and len(ctx.memo) == 1
    assert WA.window_keys(ctx, 1, "cpu")[2] == 5 + 4 + 2 + 7
