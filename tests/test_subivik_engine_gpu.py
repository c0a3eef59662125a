"""The Subivik family through the engine against the plain oracle: whole prompts, portions, decoding, mixed batches, reuse of
cache blocks and state slots, and greedy generation through the scheduler."""
import pytest
import torch

from tests import subivik_cases as cases

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
IDS = ["fp32", "bf16"]


def _run(eng, rid, toks, cuts):
    """Feeds toks in portions of the given sizes (repeating the last size); logits at every place."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        k += 1
        last = at + n == len(toks)
        out.append(eng.score_step([(rid, toks[at:at + n], list(range(n)))], [rid] if last else []))
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_whole_portions_and_decoding(name, dtype):
    """One prompt at once, in portions of many sizes (down to two tokens, across block borders), and token by token."""
    n = 75
    eng, toks, want = cases.engine(name, dtype), cases.tokens(name, n), cases.expected(name, n)
    got = {}
    for label, cuts in {"whole": [n], "one by one": [1], "two": [2], "uneven": [16, 3, 2, 17, 1, 2, 13, 5],
                        "then decode": [61, 1]}.items():
        got[label] = _run(eng, label, toks, cuts)
        cases.check(got[label], want, dtype)
    if dtype == torch.float32:
        for label in got:
            assert float(cases.error(got[label], got["whole"]).max()) < 2e-5, label
    assert len(eng.scheduler.block_manager.free_blocks) == 40
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", ["odd", "even", "between", "ones"])
def test_mixed_batches_and_reuse(name, dtype):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, and a pool so small that blocks
    and slots change hands; every request must come out as it does alone."""
    eng = cases.engine(name, dtype, num_kv_blocks=11, max_num_seqs=3)
    lens = {"a": 75, "b": 33, "c": 1, "d": 50, "e": 18}
    toks = {r: cases.tokens(name, n, seed=i) for i, (r, n) in enumerate(lens.items())}
    plan = [[("a", 3)], [("a", 30), ("b", 2)], [("b", 16), ("a", 1), ("c", 1)], [("a", 1), ("b", 1)],
            [("d", 40), ("b", 14)], [("a", 25), ("d", 1)], [("a", 1)], [("d", 1), ("a", 13), ("e", 2)],
            [("e", 1), ("a", 1), ("d", 7)], [("d", 1), ("e", 15)]]
    at, got = {r: 0 for r in lens}, {r: [] for r in lens}
    for step in plan:
        entries, end = [], []
        for r, n in step:
            entries.append((r, toks[r][at[r]:at[r] + n], list(range(n))))
            at[r] += n
            if at[r] == lens[r]:
                end.append(r)
        rows = eng.score_step(entries, end)
        for r, n in step:
            got[r].append(rows[:n])
            rows = rows[n:]
    assert at == lens and len(eng.scheduler.block_manager.free_blocks) == 11
    for i, (r, n) in enumerate(lens.items()):
        cases.check(torch.cat(got[r]), cases.expected(name, n, i), dtype)
    eng.exit()


def test_some_wanted_and_stale_slots():
    """Logits of chosen places only; then the state and cache of a request that ended are poisoned, and the next owner must
    not see them."""
    eng = cases.engine("odd", torch.float32, num_kv_blocks=5, max_num_seqs=1)
    toks, want = cases.tokens("odd", 75), cases.expected("odd", 75)
    assert eng.score_step([("a", toks[:20], [])]).shape[0] == 0
    assert eng.score_step([("a", toks[20:21], [])]).shape[0] == 0
    cases.check(eng.score_step([("a", toks[21:40], [18, 0, 7])]), want[[39, 21, 28]], torch.float32)
    cases.check(eng.score_step([("a", toks[40:41], [0])], ["a"]), want[40:41], torch.float32)
    for cuts in ([33], [1], [2, 5]):
        for pool in eng.model_runner.pools:
            pool.fill_(1e4)
        cases.check(_run(eng, "b", cases.tokens("odd", 33, seed=1), cuts), cases.expected("odd", 33, 1), torch.float32)
    eng.exit()


def test_residual_layer_by_layer():
    """The residual stream after every layer."""
    from oracle import subivik_oracle as oracle
    cfg, w = cases.model("odd")
    toks, want, got = cases.tokens("odd", 40), [], []
    oracle.forward(cfg, w, toks, per_layer=want)
    eng = cases.engine("odd", torch.float32, enforce_eager=True)
    eng.model_runner.model.layer_probe = lambda i, x: got.append(x.double().cpu())
    eng.score_step([("a", toks, [0])], ["a"])
    assert len(got) == len(want)
    for g, x in zip(got, want):
        assert float((g - x).abs().max() / x.abs().max()) < 3e-5
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding(dtype):
    """Two hundred decoded tokens after a short prompt, through block borders and every chunk, in the captured graph."""
    n = 215
    eng, toks, want = cases.engine("even", dtype), cases.tokens("even", n), cases.expected("even", n)
    cases.check(_run(eng, "a", toks, [9, 1]), want, dtype)
    cases.check(_run(eng, "b", toks, [200, 1]), want, dtype)
    eng.exit()


def _greedy_ok(prompt, got, name):
    """Each generated token is the oracle's argmax after the same prefix, or one that the oracle cannot tell from it."""
    from oracle import subivik_oracle as oracle
    cfg, w = cases.model(name)
    logits = oracle.forward(cfg, w, prompt + got[:-1], torch.float32)
    for i, t in enumerate(got):
        row = logits[len(prompt) - 1 + i]
        assert float(row.max() - row[t]) < 1e-3, f"token {i}"


@pytest.mark.parametrize("chunked", [False, True], ids=["waves", "mixed"])
def test_greedy_generation(chunked):
    """LLMEngine.generate with more requests than slots, prompts longer than the token budget (mixed steps), a prompt of one
    token, and a pool that forces preemption."""
    from minivllm_b200.engine.sequence import SamplingParams
    name, lens = "odd", [40, 1, 23, 64, 2, 17]
    prompts = [cases.tokens(name, n, seed=20 + i) for i, n in enumerate(lens)]
    outs = []
    for eager, blocks in ((False, 40), (True, 9)):
        eng = cases.engine(name, torch.float32, chunked_prefill=chunked, num_kv_blocks=blocks, enforce_eager=eager,
                           max_num_batched_tokens=24 if chunked else 128, max_num_seqs=3)
        outs.append(eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))["token_ids"])
        assert len(eng.scheduler.block_manager.free_blocks) == blocks
        eng.exit()
    for p, a, b in zip(prompts, *outs):
        assert len(a) == 12 and len(b) == 12
        _greedy_ok(p, a, name)
        _greedy_ok(p, b, name)


def test_sampled_generation_in_bf16_from_seeded_weights():
    from minivllm_b200.engine.llm_engine import LLMEngine
    from minivllm_b200.engine.sequence import SamplingParams
    eng = LLMEngine({**cases.even(), "dtype": torch.bfloat16, "seed": 5, "block_size": 64, "num_kv_blocks": 8, "max_num_seqs": 2,
                     "max_model_length": 128, "max_num_batched_tokens": 32, "chunked_prefill": True, "greedy": False})
    prompts = [cases.tokens("even", n, seed=n) for n in (50, 3)]
    out = eng.generate(prompts, SamplingParams(temperature=0.8, max_tokens=9, ignore_eos=True))["token_ids"]
    assert [len(o) for o in out] == [9, 9] and all(0 <= t < 320 for o in out for t in o)
    eng.exit()


def test_command_line_and_trace_from_a_folder(tmp_path, capsys):
    """A model folder through the command line and through the trace runner."""
    import json
    import struct

    import numpy as np

    from minivllm_b200 import _cabi, trace
    from minivllm_b200.__main__ import main
    cfg, w = cases.model("parallel_only")
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    index, data = {}, b""
    for name, t in w.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        index[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    head = json.dumps(index).encode()
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + data)
    prompt = cases.tokens("parallel_only", 20)
    main(["--model", str(tmp_path), "--prompt", ",".join(map(str, prompt)), "--max-tokens", "5", "--dtype", "float32"])
    got = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert len(got) == 5
    _greedy_ok(prompt, got, "parallel_only")
    eng = trace.make_engine(str(tmp_path), "float32", 128)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:13], "want": [12, 3]}]},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[13:], "want": [6]}], "end": ["x"]}]
    said = []
    trace.replay(eng, (json.dumps(s) for s in steps), str(tmp_path), said.append)
    eng.exit()
    assert said == ["done 0", "done 1"]
    want = cases.expected("parallel_only", 20)
    for step, rows in ((0, [12, 3]), (1, [19])):
        rows_got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), -1).copy())
        cases.check(rows_got, want[rows], torch.float32)
    _cabi.use_library(_cabi.LIB_PATH)
