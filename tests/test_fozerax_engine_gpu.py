"""The Fozerax family through the engine against the plain oracle: whole prompts, portions, decoding, mixed batches,
reuse of cache blocks and state slots, and greedy generation through the scheduler."""
import pytest
import torch

from tests import fozerax_cases as cases

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
IDS = ["fp32", "bf16"]


def _run(eng, rid, toks, cuts, end=True):
    """Feeds toks in portions of the given sizes (repeating the last size); logits at every place."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        k += 1
        last = at + n == len(toks)
        out.append(eng.score_step([(rid, toks[at:at + n], list(range(n)))], [rid] if last and end else []))
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
    """Unequal requests in one batch, portions beside single tokens, requests that pause, and a pool so small that
    blocks and slots change hands; every request must come out as it does alone."""
    eng = cases.engine(name, dtype, num_kv_blocks=11, max_num_seqs=3)
    lens = {"a": 75, "b": 33, "c": 1, "d": 50, "e": 18}
    toks = {r: cases.tokens(name, n, seed=i) for i, (r, n) in enumerate(lens.items())}
    want = {r: cases.expected(name, n, i) for i, (r, n) in enumerate(lens.items())}
    plan = [[("a", 3)], [("a", 30), ("b", 2)], [("b", 16), ("a", 1), ("c", 1)], [("a", 1), ("b", 1)],
            [("d", 40), ("b", 14)], [("a", 25), ("d", 1)], [("a", 1)], [("d", 1), ("a", 13), ("e", 2)],
            [("e", 1), ("a", 1), ("d", 7)], [("d", 1), ("e", 15)]]
    at = {r: 0 for r in lens}
    got = {r: [] for r in lens}
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
    for r in lens:
        cases.check(torch.cat(got[r]), want[r], dtype)
    eng.exit()


def test_nothing_wanted_and_some_wanted():
    eng, toks, want = cases.engine("odd", torch.float32), cases.tokens("odd", 75), cases.expected("odd", 75)
    assert eng.score_step([("a", toks[:20], [])]).shape[0] == 0
    assert eng.score_step([("a", toks[20:21], [])]).shape[0] == 0
    cases.check(eng.score_step([("a", toks[21:40], [18, 0, 7])]), want[[39, 21, 28]], torch.float32)
    cases.check(eng.score_step([("a", toks[40:41], [0])]), want[40:41], torch.float32)
    eng.exit()


def test_stale_slot_is_not_read():
    """The state and cache of a request that ended are poisoned; the next owner must not see them."""
    eng = cases.engine("odd", torch.float32, num_kv_blocks=5, max_num_seqs=1)
    a, b = cases.tokens("odd", 75), cases.tokens("odd", 33, seed=1)
    _run(eng, "a", a, [40, 1])
    for pool in eng.model_runner.pools:
        pool.fill_(1e4)
    for cuts in ([33], [1], [2, 5]):
        cases.check(_run(eng, "b", b, cuts), cases.expected("odd", 33, 1), torch.float32)
    eng.exit()


def test_layers_one_by_one():
    """The residual stream after every layer."""
    from oracle import fozerax_oracle as oracle
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


def test_long_decoding():
    """Two hundred decoded tokens after a short prompt, through block borders, in the captured decode graph."""
    n = 215
    eng, toks, want = cases.engine("even", torch.float32), cases.tokens("even", n), cases.expected("even", n)
    cases.check(_run(eng, "a", toks, [9, 1]), want, torch.float32)
    eng.exit()


def _greedy_ok(prompt, got, name):
    """Each generated token is the oracle's argmax after the same prefix, or one that the oracle cannot tell from it."""
    from oracle import fozerax_oracle as oracle
    cfg, w = cases.model(name)
    logits = oracle.forward(cfg, w, prompt + got[:-1], torch.float32)
    for i, t in enumerate(got):
        row = logits[len(prompt) - 1 + i]
        assert float(row.max() - row[t]) < 1e-3, f"token {i}"


@pytest.mark.parametrize("chunked", [False, True], ids=["waves", "mixed"])
def test_greedy_generation(chunked):
    """LLMEngine.generate with more requests than slots, prompts longer than the token budget (mixed steps), a prompt
    of one token, and a pool that forces preemption."""
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


def test_sampled_generation_runs_in_bf16():
    from minivllm_b200.engine.sequence import SamplingParams
    eng = cases.engine("even", torch.bfloat16, greedy=False, max_num_batched_tokens=32)
    prompts = [cases.tokens("even", n, seed=n) for n in (50, 3)]
    out = eng.generate(prompts, SamplingParams(temperature=0.8, max_tokens=9, ignore_eos=True))["token_ids"]
    assert [len(o) for o in out] == [9, 9] and all(0 <= t < 320 for o in out for t in o)
    eng.exit()
