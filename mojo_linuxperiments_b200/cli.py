"""Command line: ``python -m mojo_linuxperiments_b200 <command>``.

  generate   greedy generation with any registered model (a checkpoint, or a preset with random weights)
  trace      replay given tokens step by step and write logits (also ``bin/trace_run``)
  models     list the presets and architectures"""
from __future__ import annotations

import argparse
import os
import sys


def _need_kernels(dense: bool) -> None:
    """Compile what is missing; a dense model needs only its own part of the kernel library."""
    from . import _build
    if not dense:
        _build.ensure_kernels("")
    elif os.environ.get("B200RT_KERNELS", "dense") == "dense":
        os.environ["B200RT_KERNELS"] = "dense"
        _build.ensure_kernels("dense")


def _trace_args(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a W8A8 safetensors file")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files of logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold together")


def trace(args) -> int:
    from .models import registry
    family = registry.family_at(args.model)
    if args.dtype not in family.dtypes:
        print(f"the {family.name} models have no {args.dtype} form", file=sys.stderr)
        return 3
    _need_kernels(dense=family.name == "layered")
    from .engine import trace_replay

    def emit(line):
        print(line, flush=True)
    trace_replay.run(args.model, args.dtype, args.out, args.max_tokens, sys.stdin, emit)
    return 0


def generate(args) -> int:
    import torch
    from .models import registry
    from .models.config import RuntimeConfig
    preset = args.model in registry.PRESETS
    if preset:
        cfg = registry.PRESETS[args.model]()
        family = registry.family_of(cfg)
    else:
        family = registry.family_at(args.model)
    _need_kernels(dense=family.name == "layered")
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt_ids]
    longest = max(len(p) for p in prompts) + args.max_new_tokens
    rt = RuntimeConfig.from_env(dtype=args.dtype, max_batch=len(prompts), max_seq_len=(longest + 15) // 16 * 16)
    from .engine.engine import Engine
    weights = None
    if not preset:
        cfg, weights = registry.open_model(args.model, rt, "cuda")
    eng = Engine(cfg, rt, weights=weights, seed=args.seed)
    bad = [t for p in prompts for t in p if not 0 <= t < cfg.vocab]
    if bad:
        print(f"token ids {bad[:4]} outside the vocabulary of {cfg.vocab}", file=sys.stderr)
        return 2
    eng.start_batch(len(prompts), rt.max_seq_len)
    steps = [eng.prefill([torch.tensor(p, dtype=torch.int64) for p in prompts]).tolist()]
    for _ in range(args.max_new_tokens - 1):
        steps.append(eng.decode_step().tolist())
    eng.check_status()
    for b in range(len(prompts)):
        print(",".join(str(s[b]) for s in steps))
    return 0


def models(_args) -> int:
    from .models import registry
    print("architectures of checkpoint folders:", ", ".join(registry.ARCHITECTURES))
    for name, make in registry.PRESETS.items():
        cfg = make()
        print(f"{name}: {registry.family_of(cfg).name}, width {cfg.d_model}, vocabulary {cfg.vocab}")
    return 0


def trace_main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model step by step (JSON steps on "
                                 "standard input) and write the logits of the wanted places.")
    _trace_args(ap)
    return trace(ap.parse_args(argv))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="mojo_linuxperiments_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="greedy generation")
    g.add_argument("--model", required=True, help="checkpoint folder / file, or a preset (random weights)")
    g.add_argument("--prompt-ids", nargs="+", required=True, help="comma-separated token ids, one argument per prompt")
    g.add_argument("--max-new-tokens", type=int, default=16)
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--seed", type=int, default=0, help="of a preset's random weights")
    _trace_args(sub.add_parser("trace", help="replay given tokens, write logits"))
    sub.add_parser("models", help="list presets and architectures")
    args = ap.parse_args(argv)
    return {"generate": generate, "trace": trace, "models": models}[args.cmd](args)
