"""Command line: greedy or sampled generation from a model folder, token ids in and out (no tokenizer is bundled).

    python -m minivllm_b200 --model DIR --prompt 12,7,30 [--prompt ...] [--max-tokens 64] [--temperature 0]
"""
import argparse
import json


def main(argv=None):
    ap = argparse.ArgumentParser(prog="minivllm_b200", description="Generate token ids from a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be repeated")
    ap.add_argument("--max-tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=0.0, help="0 is greedy")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--block-size", type=int, default=64)
    ap.add_argument("--max-batched-tokens", type=int, default=8192)
    ap.add_argument("--chunked-prefill", action="store_true", help="portions of prompts beside decoded tokens")
    a = ap.parse_args(argv)

    import torch
    from . import _cabi
    from .csrc import build
    from .engine.llm_engine import LLMEngine
    from .engine.registry import family_of, folder_config
    from .engine.sequence import SamplingParams

    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    config = folder_config(a.model)
    _cabi.use_library(build.build(group=family_of(config).kernels))
    config.update(dtype=getattr(torch, a.dtype), block_size=a.block_size, max_num_seqs=min(len(prompts), 256),
                  max_model_length=max(len(p) for p in prompts) + a.max_tokens,
                  max_num_batched_tokens=a.max_batched_tokens, chunked_prefill=a.chunked_prefill,
                  greedy=a.temperature == 0)
    engine = LLMEngine(config)
    out = engine.generate(prompts, SamplingParams(temperature=a.temperature, max_tokens=a.max_tokens, ignore_eos=True))
    for ids in out["token_ids"]:
        print(json.dumps(ids))
    engine.exit()


if __name__ == "__main__":
    main()
