"""``python -m onnxruntime_b200.tools.generate --model DIR --prompt-ids 5,17,3 [--prompt-ids ...]``

Generates continuations of token-id prompts with a model folder (config.json + model.safetensors) of any family the
registry knows.  Prompts of different lengths run as one batch.  Prints one JSON line per prompt.
"""
from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description="generate token ids with a decoder")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt-ids", action="append", required=True, help="comma-separated token ids; repeat for a batch")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float16", "float32"])
    ap.add_argument("--provider", default="cuda", choices=["cuda", "cpu"])
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--batch", type=int, default=8, help="requests that run at a time, at most")
    ap.add_argument("--eos-token-id", type=int, default=None)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--repetition-penalty", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=None, help="sampling with this seed (greedy without it, top-k and top-p)")
    a = ap.parse_args(argv)

    from onnxruntime_b200.models.generation import GenerationConfig, generate_requests
    from onnxruntime_b200.models.registry import load_decoder
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt_ids]
    longest = max(len(p) for p in prompts) + a.max_new_tokens
    runner = load_decoder(a.model, a.dtype, batch=min(a.batch, len(prompts)), max_len=longest,
                          provider="CUDAExecutionProvider" if a.provider == "cuda" else "CPUExecutionProvider")
    outs = generate_requests(runner, prompts, GenerationConfig(
        max_new_tokens=a.max_new_tokens, eos_token_id=a.eos_token_id, temperature=a.temperature, top_k=a.top_k, top_p=a.top_p,
        repetition_penalty=a.repetition_penalty, seed=a.seed))
    for prompt, out in zip(prompts, outs):
        print(json.dumps({"prompt": prompt, "generated": out}), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
