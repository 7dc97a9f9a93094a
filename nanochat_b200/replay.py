"""
Trace replay: feed given token ids through a model folder, step by step, and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
`entries` bring the next tokens of requests, `want` are the places among them whose logits are wanted, `end` lists
requests that are finished after the step (their pages go back). Where something is wanted the step writes
OUT/<step>.f32: little-endian float32, [wanted, vocab]. Every step prints "done <step>". Requests are `Engine`
sequences: portions take the prefill path, single tokens the captured decode step, nothing is sampled.

bfloat16 is the serving precision; float32 computes everything in true float32.
"""

import argparse
import json
import os
import sys


def run(engine, max_tokens, lines, out_dir, say):
    sequences = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for entry in step.get("entries", []):
            if entry["id"] not in sequences:
                sequences[entry["id"]] = engine.open_sequence(max_tokens)
            want = list(entry.get("want", []))
            logits = sequences[entry["id"]].extend(entry["tokens"], want)
            if want:
                parts.append(logits.float().cpu())
        if parts:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path + ".tmp", "wb") as f:
                for p in parts:
                    f.write(p.contiguous().numpy().astype("<f4").tobytes())
            os.replace(path + ".tmp", path)
        for name in step.get("end", []):
            if name in sequences:
                sequences.pop(name).close()
        engine.check()
        say(f"done {step['step']}")


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda")
    args = ap.parse_args(argv)
    os.environ["NANOCHAT_DTYPE"] = args.dtype
    import torch
    from nanochat_b200.checkpoint_manager import load_model_folder
    from nanochat_b200.engine import Engine
    if args.device == "cuda" and not torch.cuda.is_available():
        print("no CUDA device", file=sys.stderr)
        return 2
    if args.dtype == "float32":
        torch.set_float32_matmul_precision("highest")
    model, tokenizer, _ = load_model_folder(args.model, torch.device(args.device), dtype=getattr(torch, args.dtype),
                                            sequence_len=max(args.max_tokens, 1))
    engine = Engine(model, tokenizer)
    run(engine, args.max_tokens, sys.stdin, args.out, lambda text: print(text, flush=True))
    return 0
