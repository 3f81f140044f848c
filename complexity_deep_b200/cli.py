"""Command line: ``python -m complexity_deep_b200 <command>``.

    info     --model DIR                    architecture, sizes, parameter count
    generate --model DIR --prompt 1,2,3     continue a prompt of token ids (several: repeat --prompt
                                            with equal lengths); prints one line of ids per sequence
    trace    ...                            replay a trace (see complexity_deep_b200/trace.py)
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


def _parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="complexity_deep_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    info = sub.add_parser("info", help="architecture and size of a checkpoint")
    info.add_argument("--model", required=True)
    gen = sub.add_parser("generate", help="continue prompts of token ids")
    gen.add_argument("--model", required=True)
    gen.add_argument("--prompt", action="append", required=True, help="token ids with commas between them")
    gen.add_argument("--max-new-tokens", type=int, default=32)
    gen.add_argument("--greedy", action="store_true")
    gen.add_argument("--temperature", type=float, default=1.0)
    gen.add_argument("--top-k", type=int, default=50)
    gen.add_argument("--top-p", type=float, default=0.9)
    gen.add_argument("--seed", type=int, default=None)
    gen.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    sub.add_parser("trace", help="replay a trace", add_help=False)
    return ap


def parse_prompts(texts) -> list:
    prompts = [[int(t) for t in text.split(",") if t.strip()] for text in texts]
    if not prompts[0] or any(len(p) != len(prompts[0]) for p in prompts):
        raise SystemExit("prompts must be non-empty and of equal length")
    return prompts


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else list(argv)
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main
        return trace_main(argv[1:])
    args = _parser().parse_args(argv)
    if args.command == "info":
        import torch
        from .models.registry import DEFAULT_ARCHITECTURE, model_class
        config = json.loads((Path(args.model) / "config.json").read_text())
        cls = model_class(config)
        with torch.device("meta"):
            model = cls(cls.config_class.from_dict(config))
        print(json.dumps({"architecture": config.get("architecture", DEFAULT_ARCHITECTURE),
                          "class": cls.__name__, "layers": len(model.layers),
                          "parameters": sum(p.numel() for p in model.parameters())}))
        return 0
    import torch
    from .models.registry import load_model
    prompts = parse_prompts(args.prompt)
    model = load_model(args.model, device="cuda", dtype=getattr(torch, args.dtype))
    if args.seed is not None:
        torch.manual_seed(args.seed)
    out = model.generate(torch.tensor(prompts, device="cuda"), max_new_tokens=args.max_new_tokens,
                         temperature=args.temperature, top_k=args.top_k, top_p=args.top_p,
                         do_sample=not args.greedy)
    for row in out.tolist():
        print(",".join(str(t) for t in row))
    return 0
