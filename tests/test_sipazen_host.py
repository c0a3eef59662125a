"""Host side of the Sipazen family: registry, weight files, configuration checks, mixed-step scheduling."""
import json
import struct

import pytest
import torch

from minivllm_b200.engine.block_manager import BlockManager
from minivllm_b200.engine.registry import family_of, folder_config
from minivllm_b200.engine.scheduler import Scheduler
from minivllm_b200.engine.sequence import SamplingParams, Sequence
from minivllm_b200.engine.sipazen import SipazenConfig, SipazenForCausalLM
from minivllm_b200.engine.weights import DictWeights, RandomWeights, SafetensorsWeights
from oracle import sipazen_oracle as oracle
from tests import sipazen_cases as cases


def _write(path, tensors):
    names = {torch.bfloat16: "BF16", torch.int32: "I32", torch.float32: "F32"}
    index, blobs, at = {"__metadata__": {"format": "pt"}}, [], 0
    for k, t in tensors.items():
        raw = t.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        index[k] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(index).encode()
    path.write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))


def test_family_is_chosen_by_architecture(tmp_path):
    cfg, _ = cases.model("odd")
    assert family_of(cfg).model is SipazenForCausalLM
    assert family_of({}).name == "Qwen3ForCausalLM"
    with pytest.raises(ValueError, match="unknown architecture"):
        family_of({"architecture": "Nothing"})
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    c = folder_config(str(tmp_path), block_size=32)
    assert c["block_size"] == 32 and c["model_dir"] == str(tmp_path) and c["layers"] == cfg["layers"]
    (tmp_path / "config.json").write_text("{}")
    with pytest.raises(ValueError, match="names no architecture"):
        folder_config(str(tmp_path))


def test_safetensors_round_trip(tmp_path):
    g = torch.Generator().manual_seed(1)
    t = {"a": torch.randn(3, 5, generator=g).to(torch.bfloat16), "n": torch.arange(7, dtype=torch.int32),
         "f": torch.randn(2, generator=g), "one": torch.randn(1, 1, generator=g).to(torch.bfloat16)}
    _write(tmp_path / "m.safetensors", t)
    w = SafetensorsWeights(str(tmp_path / "m.safetensors"), torch.float32, "cpu")
    assert torch.equal(w("a", (3, 5)), t["a"].float()) and torch.equal(w("n", (7,)), t["n"])
    with pytest.raises(ValueError, match="shape"):
        w("f", (3,))
    with pytest.raises(KeyError):
        w("zzz", (1,))
    with pytest.raises(ValueError, match="belong to no part"):
        w.check_all_used()
    (tmp_path / "bad.safetensors").write_bytes(struct.pack("<Q", 1 << 40))
    with pytest.raises(ValueError):
        SafetensorsWeights(str(tmp_path / "bad.safetensors"), torch.float32, "cpu")


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_model_takes_exactly_the_checkpoint(name):
    cfg, w = cases.model(name)
    c = SipazenConfig.from_dict(cfg)
    m = SipazenForCausalLM(c, dtype=torch.float32, device="cpu", weights=DictWeights(w, torch.float32, "cpu"))
    assert c.widest_activation() > 0 and len(m.layers) == len(cfg["layers"])
    extra = dict(w, other=torch.zeros(1))
    with pytest.raises(ValueError, match="other"):
        SipazenForCausalLM(c, dtype=torch.float32, device="cpu", weights=DictWeights(extra, torch.float32, "cpu"))
    SipazenForCausalLM(c, dtype=torch.float32, device="cpu", weights=RandomWeights(0, torch.float32, "cpu"))


def test_configuration_errors():
    cfg, _ = cases.model("odd")
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        SipazenConfig.from_dict(bad)
    bad = json.loads(json.dumps(cfg))
    bad["norm"]["groups"] = 7
    with pytest.raises(ValueError, match="groups"):
        SipazenConfig.from_dict(bad)
    with pytest.raises(ValueError, match="one GPU"):
        SipazenForCausalLM(SipazenConfig.from_dict(cfg), tp_size=2)
    with pytest.raises(ValueError, match="chunked prefill"):
        Scheduler(4, 64, 8, 16, -1, prefix_caching=True, chunked_prefill=True)


def test_oracle_is_causal_and_sees_every_mechanism():
    """A later token changes nothing before it; changing one tensor of each mechanism changes the logits."""
    cfg, w = cases.model("odd")
    toks = cases.tokens("odd", 12)
    base = oracle.forward(cfg, w, toks)
    assert torch.equal(base[:9], oracle.forward(cfg, w, toks[:9] + [1, 2, 3])[:9])
    for name in ("l1.mix.sink", "l1.mix.g", "l0.mix.conv.b", "l0.mix.D", "l0.mix.A_log", "l0.mix.dt_bias", "l0.mix.norm",
                 "l0.mlp.router.b", "l0.mlp.shared.sg", "l0.rg1.b", "l0.rg2", "l1.norm1b", "l1.mix.dkv.norm",
                 "final.norm"):
        moved = dict(w)
        moved[name] = -w[name]
        assert float(cases.error(oracle.forward(cfg, moved, toks), base).max()) > 1e-3, name


def test_mixed_steps_cover_every_token_once():
    """Prompts beyond the token budget, decoding beside portions, preemption: the tokens of every sequence are run in
    order, exactly once per residency, and budgets hold."""
    s = Scheduler(max_num_seqs=3, max_num_batched_tokens=10, num_blocks=8, block_size=4, eos=-1, chunked_prefill=True)
    seqs = [Sequence(range(n), SamplingParams(max_tokens=6, ignore_eos=True), block_size=4) for n in (17, 1, 9, 25, 2)]
    for q in seqs:
        s.add_sequence(q)
    preempted, decode_steps = 0, 0
    for _ in range(400):
        if s.is_finished():
            break
        batch, is_prefill = s.schedule()
        assert batch and len(set(map(id, batch))) == len(batch) <= 3
        assert sum(q.num_scheduled_tokens for q in batch) <= 10
        for q in batch:
            assert 0 <= q.num_cached_tokens and q.num_cached_tokens + q.num_scheduled_tokens <= len(q)
            assert len(q.block_table) * 4 >= q.num_cached_tokens + q.num_scheduled_tokens
        assert is_prefill == any(not q.on_device for q in batch)
        decode_steps += not is_prefill
        before = {id(q): (q.num_cached_tokens, q.num_scheduled_tokens, len(q)) for q in batch}
        s.postprocess(batch, [7] * len(batch))
        for q in batch:
            c, n, l = before[id(q)]
            assert len(q) == l + (c + n == l)
        preempted += sum(not q.block_table and 0 < q.num_completion_tokens < 6 for q in seqs)
    assert s.is_finished() and decode_steps > 0 and preempted > 0
    assert all(q.num_completion_tokens == 6 for q in seqs)
    assert len(s.block_manager.free_blocks) == 8 and len(s.block_manager.free_slots) == 3


def test_mixed_lookahead_bookkeeping():
    """advance() appends nothing for a prompt in progress, and fill_tokens skips it."""
    s = Scheduler(max_num_seqs=2, max_num_batched_tokens=6, num_blocks=12, block_size=4, eos=-1, chunked_prefill=True)
    a, b = Sequence([1, 2], SamplingParams(max_tokens=3, ignore_eos=True), 4), Sequence(range(9), SamplingParams(max_tokens=3, ignore_eos=True), 4)
    s.add_sequence(a)
    s.add_sequence(b)
    batch, prefill = s.schedule()
    assert prefill and [q.num_scheduled_tokens for q in batch] == [2, 4]
    at = s.advance(batch)
    assert at == [2, -1] and len(a) == 3 and len(b) == 9 and b.num_cached_tokens == 4
    s.fill_tokens(batch, at, [11, 12])
    assert a.token_ids == [1, 2, 11] and b.token_ids == list(range(9))


def test_reserve_grows_a_table():
    bm = BlockManager(4, 4, 2)
    q = Sequence([1, 2, 3], block_size=4)
    bm.allocate(q)
    q.token_ids.extend(range(9))
    bm.reserve(q)
    assert len(q.block_table) == 3
    q.token_ids.extend(range(9))
    with pytest.raises(RuntimeError, match="no free cache block"):
        bm.reserve(q)
