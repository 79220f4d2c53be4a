"""``bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N``

Feeds given token ids through a model step by step and writes logits; nothing is sampled.  DIR holds config.json and
model.safetensors; the family is chosen by config.json.  Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch of ``PagedDecoderRunner.step``, the call that generation uses.  Logits of the wanted
places go to OUT/<step>.f32 ([wanted, vocab], little-endian float32) when there are any, then "done <step>" is printed.
``end`` lists the sequences that are finished after the step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live sequences hold at any time, at most")
    ap.add_argument("--max-sequences", type=int, default=256, help="sequences that are live at any time, at most")
    ap.add_argument("--block-size", type=int, default=128)
    a = ap.parse_args(argv)

    from onnxruntime_b200.models.registry import load_decoder
    sequences = max(1, min(a.max_sequences, a.max_tokens))
    runner = load_decoder(a.model, a.dtype, batch=sequences, max_len=a.max_tokens, max_tokens=a.max_tokens, block_size=a.block_size)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = runner.step([(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
        runner.sess.check_device_status()
        if logits.shape[0]:
            logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for seq in step.get("end", []):
            runner.release(seq)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
