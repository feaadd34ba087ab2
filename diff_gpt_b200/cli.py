"""Command line: `python -m diff_gpt_b200 generate ...` and `python -m diff_gpt_b200 trace ...` (also `bin/trace_run`).

generate   continue a prompt of token ids with a checkpoint folder (config.json, model.safetensors)
trace      replay a recorded trace of token ids step by step and write the logits it asks for
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def _load(args):
    from .model.registry import load_model

    # float32 means true 32-bit products
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    return load_model(args.model, DTYPES[args.dtype], "cuda")


def generate(args) -> int:
    from .model.engine import Engine
    from .sampler.nucleus import NucleusSampler
    from .sampler.temperature import TemperatureSampler

    sampler = TemperatureSampler(args.temperature)
    if args.top_p < 1.0:
        sampler = NucleusSampler(args.top_p, sampler)
    prompt = [int(t) for t in args.tokens.replace(",", " ").split()]
    results, _ = Engine(_load(args)).generate_batch(
        prompt, num_samples=args.num_samples, max_tokens=args.max_tokens, sampler=sampler, seed=args.seed
    )
    for r in results:
        print(" ".join(map(str, r[len(prompt) :])))
    return 0


def trace(args) -> int:
    """Steps are JSON objects, one a line, on standard input: {"step": n, "entries": [{"id", "tokens", "want"}],
    "end": [ids]}.  The wanted logits of a step go to OUT/<step>.f32 (little-endian fp32, in the order of the entries);
    `done <step>` is printed when the step is over."""
    from .model.engine import StepRunner

    runner = StepRunner(_load(args))
    for line in sys.stdin:
        if not line.strip():
            continue
        job = json.loads(line)
        outs = [runner.step(e["id"], e["tokens"], e["want"]) for e in job["entries"]]
        for request in job["end"]:
            runner.finish(request)
        outs = [o for o in outs if o.shape[0]]
        if outs:
            path = os.path.join(args.out, f"{job['step']}.f32")
            torch.cat(outs).cpu().numpy().astype("<f4").tofile(path)
        print(f"done {job['step']}", flush=True)
    return 0


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="diff_gpt_b200", description="Serve a checkpoint folder on one B200.")
    sub = ap.add_subparsers(dest="command", required=True)
    for name, fn, text in (("generate", generate, "continue a prompt of token ids"),
                           ("trace", trace, "replay a trace of token ids from standard input")):
        p = sub.add_parser(name, help=text)
        p.set_defaults(fn=fn)
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
        if name == "generate":
            p.add_argument("--tokens", required=True, help="prompt: token ids separated by spaces or commas")
            p.add_argument("--max-tokens", type=int, default=64)
            p.add_argument("--num-samples", type=int, default=1)
            p.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
            p.add_argument("--top-p", type=float, default=1.0)
            p.add_argument("--seed", type=int, default=42)
        else:
            p.add_argument("--out", required=True, help="folder for the logits")
            p.add_argument("--max-tokens", type=int, default=0,
                           help="the most tokens live at any time (caches grow on demand; accepted for sizing)")
    args = ap.parse_args(argv)
    return args.fn(args)
