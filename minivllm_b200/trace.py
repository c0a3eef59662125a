"""Replays given tokens through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

DIR holds config.json and model.safetensors.  Steps are read from standard input, one JSON object a line:

    {"step": 4, "entries": [{"id": "x", "tokens": [12, 7], "want": [1]}, {"id": "y", "tokens": [30], "want": []}],
     "end": ["y"]}                    (in one line)

`want` names places among an entry's own tokens; `end` lists requests that are over.  Each step's entries run as one
batch through `LLMEngine.score_step`, i.e. the engine's own cache blocks, state slots, model step and (for single
tokens) decode graph.  The logits at the wanted places go to OUT/<step>.f32, little-endian 32-bit floats in the order
of the entries, and a line `done <step>` follows every step.  `--max-tokens` sizes the cache pool, in tokens of all
requests that are running at once, whole blocks each.
"""
import argparse
import json
import os
import sys

BLOCK = 64
LIVE = 4


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay given tokens through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the cache pool in tokens")
    return ap.parse_args(argv)


def make_engine(model, dtype, max_tokens):
    import torch
    from . import _cabi
    from .csrc import build
    from .engine.llm_engine import LLMEngine
    from .engine.registry import family_of, folder_config

    config = folder_config(model)
    _cabi.use_library(build.build(group=family_of(config).kernels))
    blocks = max(1, -(-max_tokens // BLOCK))
    config.update(dtype=getattr(torch, dtype), block_size=BLOCK, num_kv_blocks=blocks, max_num_seqs=LIVE,
                  max_model_length=blocks * BLOCK, max_num_batched_tokens=blocks * BLOCK, chunked_prefill=True,
                  greedy=True, keep_logits=True)
    return LLMEngine(config)


def replay(engine, lines, out, say):
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        logits = engine.score_step(entries, step.get("end", []))
        if logits.shape[0]:
            path = os.path.join(out, f"{step['step']}.f32")
            logits.numpy().astype("<f4").tofile(path + ".part")
            os.replace(path + ".part", path)
        say(f"done {step['step']}")


def main(argv=None):
    args = parse_args(argv)
    engine = make_engine(args.model, args.dtype, args.max_tokens)
    replay(engine, iter(sys.stdin.readline, ""), args.out, lambda s: print(s, flush=True))
    engine.exit()
    return 0
