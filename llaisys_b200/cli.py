"""Command line of the package, for any model of the registry:

    python -m llaisys_b200 info --model DIR
    python -m llaisys_b200 generate --model DIR --prompt 12,7,99 [--prompt ...] --max-new-tokens 32

Prompts are token ids (there is no tokenizer in the package). Greedy prompts run together through the batching engine;
with --top-k other than 1 each is sampled on its own. One JSON line per prompt.
"""
from __future__ import annotations

import argparse
import json
from pathlib import Path

from .libllaisys import DeviceType
from .models import load_model, model_class
from .models.base import DTYPE_NAMES
from .serving import Engine


def _tokens(text: str) -> list[int]:
    return [int(t) for t in text.replace(",", " ").split()]


def _generate(args) -> int:
    device = {"auto": None, "cpu": DeviceType.CPU, "nvidia": DeviceType.NVIDIA}[args.device]
    kwargs = {} if args.dtype == "auto" else {"dtype": DTYPE_NAMES[args.dtype]}
    model = load_model(args.model, device, **kwargs)
    prompts = args.prompt
    longest = max(len(p) for p in prompts) + args.max_new_tokens
    if args.top_k == 1:
        model.configure_cache(min(len(prompts), args.max_batch), longest)
        engine = Engine(model, max_batch=min(len(prompts), args.max_batch), max_tokens_per_step=args.max_tokens_per_step,
                        prefill_chunk=args.prefill_chunk)
        done = engine.run([(0, p, args.max_new_tokens) for p in prompts])
        engine.close()
    else:
        model.configure_cache(1, longest)
        done = {i: model.generate(p, args.max_new_tokens, args.top_k, args.top_p, args.temperature, args.seed)[len(p):]
                for i, p in enumerate(prompts)}
    for i, p in enumerate(prompts):
        print(json.dumps({"prompt": p, "tokens": done[i]}))
    return 0


def _info(args) -> int:
    config = json.loads((Path(args.model) / "config.json").read_text())
    print(json.dumps({"class": model_class(config).__name__, "config": config}))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m llaisys_b200", description=__doc__,
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    gen = sub.add_parser("generate", help="continue prompts of token ids")
    gen.add_argument("--model", required=True, help="checkpoint directory (config.json + *.safetensors)")
    gen.add_argument("--prompt", required=True, action="append", type=_tokens, help="token ids, e.g. 12,7,99 (repeatable)")
    gen.add_argument("--max-new-tokens", type=int, default=32)
    gen.add_argument("--device", default="auto", choices=["auto", "cpu", "nvidia"])
    gen.add_argument("--dtype", default="auto", choices=["auto", *DTYPE_NAMES])
    gen.add_argument("--top-k", type=int, default=1, help="1 = greedy")
    gen.add_argument("--top-p", type=float, default=0.8)
    gen.add_argument("--temperature", type=float, default=0.8)
    gen.add_argument("--seed", type=int, default=None)
    gen.add_argument("--max-batch", type=int, default=64)
    gen.add_argument("--max-tokens-per-step", type=int, default=4096)
    gen.add_argument("--prefill-chunk", type=int, default=512)
    gen.set_defaults(run=_generate)
    info = sub.add_parser("info", help="which class a checkpoint selects")
    info.add_argument("--model", required=True)
    info.set_defaults(run=_info)
    args = ap.parse_args(argv)
    return args.run(args)
