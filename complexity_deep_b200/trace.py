"""Replays a trace of token ids through a model and writes the logits that it asks for.

Steps arrive as JSON lines ``{"step", "entries": [{"id", "tokens", "want"}], "end": [ids]}``: every
entry continues (or starts) the request `id` with its next tokens from the state that earlier steps
left; `want` lists the places among them whose logits are written to ``<out>/<step>.f32``
(little-endian fp32, [wanted, vocab]); requests in `end` give their state back.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

REFUSED = 3      # exit code: the model does not run in the requested precision


def _parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__)
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0,
                    help="most tokens that live requests hold at any time")
    return ap


class TraceReplay:
    def __init__(self, model, device) -> None:
        self.model, self.device = model, device
        self.pool = model.state_pool()

    def step(self, entries, end):
        """Runs one step; returns the wanted logits as fp32 [wanted, vocab] on the CPU, or None."""
        import torch
        rows = []
        for e in entries:
            ids = torch.tensor([e["tokens"]], dtype=torch.int64, device=self.device)
            want = torch.tensor(e["want"], dtype=torch.int64, device=self.device)
            out = self.model(ids, past_key_values=self.pool.get(e["id"]), use_cache=True, logit_rows=want)
            if e["want"]:
                rows.append(out.logits.float().cpu())
        for request in end:
            self.pool.release(request)
        return torch.cat(rows, 0) if rows else None


def main(argv=None) -> int:
    args = _parser().parse_args(argv)
    import torch
    from . import ops
    from .models.registry import load_model, model_class

    config = json.loads((Path(args.model) / "config.json").read_text())
    cls = model_class(config)
    if not hasattr(cls, "state_pool"):
        print(f"{cls.__name__} keeps no per-request state", file=sys.stderr)
        return REFUSED if args.dtype == "float32" else 1
    if not torch.cuda.is_available():
        raise RuntimeError("a CUDA device is needed; there is no CPU path")
    model = load_model(args.model, device="cuda", dtype=getattr(torch, args.dtype))
    replay = TraceReplay(model, torch.device("cuda"))
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end", []))
        if logits is not None:
            logits.numpy().astype("<f4").tofile(Path(args.out) / f"{s['step']}.f32")
        torch.cuda.synchronize()
        print(f"done {s['step']}", flush=True)
    ops.status_fetch()
    return 0
