"""Trace replay: given token ids go through a model step by step, through the engine that serves it, and the logits that
the trace asks for are written out. Nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

DIR holds config.json and model.safetensors; the model class comes from the registry. Steps are read from standard input,
one JSON object a line:

    {"step": 4, "entries": [{"id": "q7", "tokens": [11, 2], "want": [1]}, {"id": "q9", "tokens": [8], "want": []}], "end": ["q7"]}

All entries of a step are one batch. ``want`` lists places among an entry's tokens; their logits go to OUT/<step>.f32
(little-endian fp32 [wanted, vocab], entry order). A request is admitted at its first entry and gives back its pages and
slot when an ``end`` names it. After every step ``done <step>`` is printed. The cache holds N tokens (in whole pages) and
four sequences.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4
BLOCK = 16


class TraceReplay:
    def __init__(self, engine):
        self.engine = engine
        self.live = {}

    def run_step(self, step: dict):
        """fp32 logits [wanted, vocab] as a numpy array, or None when nothing is wanted."""
        entries, want = [], []
        for e in step.get("entries", []):
            rid = e["id"]
            if rid not in self.live:
                self.live[rid] = self.engine.open()
            entries.append((self.live[rid], [int(t) for t in e["tokens"]]))
            want.append([int(k) for k in e.get("want", [])])
        logits = self.engine.execute(entries, want)
        out = logits.float().cpu().numpy() if logits is not None else None
        for rid in step.get("end", []):
            seq = self.live.pop(rid, None)
            if seq is not None:
                self.engine.close(seq)
        return out


def make_replay(folder: str, dtype, device, max_tokens: int) -> TraceReplay:
    from ..models.registry import load_pretrained
    from ..models.scheduler import EngineConfig
    from . import make_engine
    blocks = (max_tokens + BLOCK - 1) // BLOCK
    model = load_pretrained(folder, dtype, device)
    engine = make_engine(model, EngineConfig(block_size=BLOCK, num_blocks=blocks, max_seq_len=blocks * BLOCK,
                                             max_batch_size=MAX_LIVE))
    if not hasattr(engine, "execute"):
        raise SystemExit("trace_run: this model's engine does not take given schedules")
    return TraceReplay(engine)


def replay(rep: TraceReplay, lines, out_dir: str, done) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = rep.run_step(step)
        if logits is not None:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(logits.astype("<f4").tobytes())
            os.replace(path + ".part", path)
        done(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)

    import torch

    from .. import _native, build
    from ..models.registry import read_config, resolve
    if not torch.cuda.is_available():
        print("trace_run: no CUDA GPU is visible", file=sys.stderr)
        return 1
    kernels = resolve(read_config(os.path.join(a.model, "config.json"))).kernels
    _native.use_library(build.ensure(kernels) if kernels else build.build_cuda())
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.cuda.set_device(0)
    rep = make_replay(a.model, getattr(torch, a.dtype), torch.device("cuda", 0), a.max_tokens)
    os.makedirs(a.out, exist_ok=True)

    def done(text):
        print(text, flush=True)
    replay(rep, iter(sys.stdin.readline, ""), a.out, done)
    status = _native.read_status(torch.cuda.current_stream().cuda_stream)
    if status != 0:
        print(f"trace_run: a kernel reported status {status}", file=sys.stderr)
        return 1
    return 0
