"""
Serving benchmark of a model that is served only (Lupodra, Safepel) beside GPT at equal width and depth, random weights:

    python -m scripts.serve_bench                        # Lupodra, every size below
    python -m scripts.serve_bench --model Safepel --sizes d12 --batch-sizes 1,8
    python bench.py --serve Safepel                      # the same, every size

Per size and model: prefill tokens/s of a prompt (device time of the prompt pass: CUDA events around it, median of
several, a write larger than L2 before each) and tokens/s of decoding through `Engine.generate` at several batch
sizes. Then, per kernel of the new model, its distance from the roofline beside the like kernel of GPT
(`nanochat_b200.ops.microbench serve`). The last line is one JSON object.
"""
import argparse
import json
import os
import statistics

import torch

from nanochat_b200.common import compute_init
from nanochat_b200.engine import Engine
from scripts.infer_bench import _SyntheticTokenizer, bench_generate

# name -> (width, layers): d12 and d26 are the depths GPT is quoted at, "wide" a few layers of a larger model's width
SIZES = {"d12": (768, 12), "d26": (1664, 26), "wide": (4096, 6)}
VOCAB = 32768


def lupodra_config(width, layers, window=512):
    """Layers shaped like a real model's: 128-dim heads with 64 rotated dimensions, a 512-entry latent, dense and expert
    feed-forwards in turn, 4 of 16 experts of one width each."""
    mixer = {"heads": width // 128, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": -(-width * 3 // 4 // 64) * 64,
             "scale": 192 ** -0.5, "rot": {"base": 10000.0, "dims": 64}, "mask": {"size": window}}
    dense = {"kind": "dense", "ff": 4 * width}
    moe = {"kind": "moe", "expert": {"ff": width}, "router": {"experts": 16, "top": 4}}
    return {"architecture": "Lupodra", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 0.7, "loop": None,
            "layers": [{"type": "latent_attention", "mixer": mixer, "mlp": moe if i % 2 else dense} for i in range(layers)]}


def safepel_config(width, layers, window=512):
    """Delta layers (as many 128-dim value heads as GPT has heads, half as many key heads) and parallel ones (half the heads
    attend to a window, half decay) in turn, gated feed-forwards of 8/3 width: 12 width^2 weights a layer, as GPT has."""
    heads = width // 128
    keys = max(k for k in range(1, heads // 2 + 1) if heads % k == 0)
    ff = -(-width * 8 // 3 // 64) * 64
    delta = {"heads": heads, "kv_heads": keys, "dim": 128, "vdim": 128, "conv": 4}
    a, b = heads - heads // 2, heads // 2
    left = {"heads": a, "kv_heads": 1, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 20.0, "rot": {"base": 10000.0, "dims": 128}, "mask": {"size": window}}
    right = {"heads": b, "dim": 128, "vdim": 128, "decay": [1 - 2.0 ** -(2 + 6 * i / b) for i in range(b)]}
    parallel = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}
    kinds = [("delta", delta), ("parallel", parallel)]
    return {"architecture": "Safepel", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "layers": [{"type": kinds[i % 2][0], "mixer": kinds[i % 2][1], "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)]}


CONFIGS = {"Lupodra": lupodra_config, "Safepel": safepel_config}


def build(kind, width, layers, device):
    from nanochat_b200.models.registry import get_architecture
    arch = get_architecture(kind)
    if kind == "GPT":
        config = arch.config_from_dict(dict(sequence_len=4096, vocab_size=VOCAB, n_layer=layers, n_head=width // 128, n_kv_head=width // 128,
                                            n_embd=width, window_pattern="SSSL"))
        return arch.build(config, device)
    return arch.build(arch.config_from_dict(CONFIGS[kind](width, layers), sequence_len=4096), device)


def prefill_ms(engine, prompt, iters=7):
    """Median device milliseconds of the prompt pass with the last position's logits."""
    device = engine.model.get_device()
    ids = torch.tensor([prompt], device=device)
    cache = engine._pooled_cache(1, len(prompt), len(prompt) + 1)
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=device)
    times = []
    with torch.inference_mode():
        for i in range(iters + 3):
            view = cache.begin_prompt(len(prompt))
            flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            engine._prompt_logits(ids, view, [len(prompt) - 1])
            b.record()
            torch.cuda.synchronize()
            if i >= 3:
                times.append(a.elapsed_time(b))
    cache.in_use = False
    return statistics.median(times)


def run(sizes, batch_sizes, prompts, decode_tokens, kinds):
    _, _, _, _, device = compute_init("cuda")
    tok = _SyntheticTokenizer(VOCAB)
    out = []
    for name in sizes:
        width, layers = SIZES[name]
        for kind in kinds:
            model = build(kind, width, layers, device)
            engine = Engine(model, tok)
            g = torch.Generator().manual_seed(0)
            row = {"size": name, "width": width, "layers": layers, "model": kind, "prefill": {}, "decode": {}}
            for n in prompts:
                prompt = torch.randint(0, VOCAB - 9, (n,), generator=g).tolist()
                ms = prefill_ms(engine, prompt)
                row["prefill"][n] = {"ms": round(ms, 3), "tok_per_sec": round(n / ms * 1e3), "tflops": round(model.estimate_prefill_flops(n) / ms / 1e9, 1)}
            prompt = torch.randint(0, VOCAB - 9, (512,), generator=g).tolist()
            for bs in batch_sizes:
                bench_generate(engine, prompt, bs, 8, 1.0, 50)
                times = bench_generate(engine, prompt, bs, decode_tokens, 1.0, 50)["step_times"]
                if times:
                    row["decode"][bs] = {"tpot_ms": round(1e3 * statistics.median(times), 3), "tok_per_sec": round(bs * len(times) / sum(times), 1)}
            engine.check()
            print(json.dumps(row), flush=True)
            out.append(row)
            del model, engine
            torch.cuda.empty_cache()
    return out


def main(argv=None):
    ap = argparse.ArgumentParser(description="Serving benchmark of a served model beside GPT")
    ap.add_argument("--model", default="Lupodra", choices=sorted(CONFIGS))
    ap.add_argument("--alone", action="store_true", help="skip GPT")
    ap.add_argument("--sizes", default=",".join(SIZES))
    ap.add_argument("--batch-sizes", default="1,8,32")
    ap.add_argument("--prompts", default="512,2048")
    ap.add_argument("--decode-tokens", type=int, default=64)
    ap.add_argument("--no-kernels", action="store_true", help="skip the per-kernel comparison")
    args = ap.parse_args(argv)
    ints = lambda s: [int(x) for x in s.split(",") if x]
    kinds = (args.model,) if args.alone else (args.model, "GPT")
    rec = {"metric": f"serving throughput, {args.model} beside GPT", "data": "synthetic, random weights", "dtype": "bf16",
           "rows": run(args.sizes.split(","), ints(args.batch_sizes), ints(args.prompts), args.decode_tokens, kinds)}
    if not args.no_kernels:
        from nanochat_b200.ops.microbench import SERVE
        rec["kernels"] = SERVE[args.model]()
    if os.path.exists("MEASURED_PEAKS.json"):
        with open("MEASURED_PEAKS.json") as f:
            rec["measured_peaks"] = {k: v for k, v in json.load(f).items() if k in ("hbm_gbs", "bf16_tflops")}
    print(json.dumps(rec))


if __name__ == "__main__":
    main()
