"""Trace replay: feeds given token ids through a model step by step and writes the logits asked for.

Steps come as JSON lines on standard input,
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [0, 1]}], "end": []}
each entry appending its tokens to the request's sequence; ``end`` names requests that are finished after the step.
A step in which something is wanted leaves <out>/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of
the entries and of ``want``); after every step a line "done <step>" is printed.  The requests occupy slots of a
running batch of the same runtime that ``CausalTransformer.generate`` and the serving loops drive.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from . import registry


class TraceRunner:
    def __init__(self, network, slots: int):
        self.rt = network._runtime(slots, 1)
        self.slots = {}                       # request id -> slot
        self.free = list(range(slots))[::-1]
        self.rt.start_batch(slots)

    def step(self, step: dict):
        """Runs one step; returns the logits [wanted, vocab] on the CPU, or None."""
        out = []
        for e in step["entries"]:
            if e["id"] not in self.slots:
                if not self.free:
                    raise RuntimeError("more live requests than slots")
                self.slots[e["id"]] = self.free.pop()
            if e["tokens"]:
                tokens = torch.tensor(e["tokens"], dtype=torch.int32, device=self.rt.device)
                out.append(self.rt.extend(self.slots[e["id"]], tokens, e.get("want", ())))
        for name in step.get("end", ()):
            slot = self.slots.pop(name, None)
            if slot is not None:
                self.rt.release(slot)
                self.free.append(slot)
        self.rt.check_device_status()
        out = [o for o in out if o.shape[0]]
        return torch.cat(out).cpu() if out else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids through a model")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=1, help="most requests that are live at any time")
    args = ap.parse_args(argv)
    net = registry.load_network(args.model, mtj_dtype=args.dtype, seq=max(2, args.max_tokens))
    runner = TraceRunner(net, args.slots)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = runner.step(step)
        if logits is not None:
            logits.numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    net.close()
    return 0
