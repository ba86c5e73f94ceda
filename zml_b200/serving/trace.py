"""Replays a trace of given token ids through the engine and writes the logits that the trace asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Steps come on standard input, one JSON object a line:

    {"step": 7, "entries": [{"id": "x", "tokens": [41, 8], "want": [1]}, {"id": "y", "tokens": [12], "want": []}], "end": ["y"]}

The entries of a step are one batch (`Engine.step`): each brings its request's next tokens and the places among them whose
logits are wanted; a request is admitted at its first entry.  `end` names the requests that are finished after the step:
their pages and state slots are free again.  Wanted logits go to DIR/<step>.f32 (float32, [wanted, vocab]); behind every
step a line `done <step>` is printed.  The cache holds --max-tokens tokens (in pages of 64) and four requests.

Exit code 3: the model's family has no fp32 kernels on the GPU and --dtype float32 was asked for.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
MAX_LIVE = 4


def build_engine(model_dir: str, dtype_name: str, max_tokens: int, device: str):
    import torch

    from .. import _build
    from ..models import common, hub
    from ..models.registry import model_class_for
    from ..ops import _lib
    from .engine import Engine
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype_name]
    _, model_cls = model_class_for(common.read_config_json(model_dir))
    if device == "cuda":
        if dtype == torch.float32 and not model_cls.FP32_ON_GPU:
            print(f"{model_cls.__name__} has no fp32 kernels", file=sys.stderr)
            raise SystemExit(3)
        if "ZB_CUDA_LIB" not in os.environ:
            _lib.use(_build.ensure_cuda(model_cls.KERNEL_SOURCES))
    model, _ = hub.load_model(model_dir, device=device, dtype=dtype)
    pages = (max_tokens + PAGE - 1) // PAGE
    return Engine(model, num_pages=pages + 1, page_size=PAGE, max_batch=MAX_LIVE, max_seq_len=pages * PAGE, num_state_slots=MAX_LIVE)


class Replay:
    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.live: dict = {}

    def run(self, step: dict) -> None:
        entries, want = [], []
        for e in step["entries"]:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open_request()
            entries.append((self.live[e["id"]], e["tokens"]))
            want.append(e.get("want", []))
        lg = self.engine.step(entries, want) if entries else None
        if lg is not None:
            lg.float().cpu().numpy().astype("<f4").tofile(os.path.join(self.out_dir, f"{step['step']}.f32"))
        for i in step.get("end", []):
            self.engine.release(self.live.pop(i))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    args = ap.parse_args(argv)
    replay = Replay(build_engine(args.model, args.dtype, args.max_tokens, args.device), args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        replay.run(step)
        print(f"done {step['step']}", flush=True)
    if args.device == "cuda":
        from .. import ops
        ops.raise_on_status()
    return 0
