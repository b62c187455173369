"""Replays a trace: steps of given tokens go through a model's forward, cache manager and state slots exactly
as an engine's steps do, and the logits that are asked for are written out. Nothing is sampled.

Each input line is a JSON object for one step, here the eighth, which runs two requests and ends one::

    {"step": 7, "entries": [{"id": "x", "tokens": [11, 4], "want": [1]}, {"id": "y", "tokens": [9], "want": []}], "end": ["y"]}

An entry continues a request with ``tokens``; ``want`` indexes those of them whose logits go to ``<out>/<step>.f32``
(little-endian f32, a row per index, in the order given; no file when no entry wants any). ``end`` releases the
blocks and state slots of requests. Once a step has run, ``done <step>`` is printed."""
from __future__ import annotations

import argparse
import json
import os
import sys

from . import engine
from .backend import CudaBackend
from .registry import load_model
from .types import DType, ForwardBatch

BLOCK = 16
ROUND = 64  # the capacity is given in units of this many tokens
STATE_SLOTS = 4


class TraceRunner:
    """The live requests of a trace, their block tables and state slots, and the model they run on."""

    def __init__(self, model):
        self.model = model
        self.slots = model.num_state_slots()
        self.cache = engine.KvCacheManager(model.num_blocks, model.block_size, False, num_state_slots=self.slots)
        self.live = {}  # request -> (sequence id, tokens so far)
        self.next_id = 1

    @classmethod
    def from_directory(cls, directory: str, dtype: DType, max_tokens: int) -> "TraceRunner":
        blocks = (max_tokens + ROUND - 1) // ROUND * (ROUND // BLOCK)
        return cls(load_model(directory, blocks, BLOCK, CudaBackend(0), compute_dtype=dtype, max_batch_tokens=blocks * BLOCK,
                              max_batch_sequences=STATE_SLOTS, num_state_slots=STATE_SLOTS))

    def step(self, entries, end=()):
        """Runs one batch; returns the wanted logits [wanted, vocab] or None when nothing is wanted."""
        tokens, positions, ids, counts, ctx, tables, rows = [], [], [], [], [], [], []
        for e in entries:
            new = e["tokens"]
            if not new:
                continue
            if e["id"] in self.live:
                sid, done = self.live[e["id"]]
                self.cache.extend(sid, len(new))
            else:
                sid, done = self.next_id, 0
                self.next_id += 1
                self.cache.allocate(sid, new)
            self.live[e["id"]] = (sid, done + len(new))
            rows += [len(tokens) + w for w in e.get("want", ())]
            tokens += new
            positions += range(done, done + len(new))
            ids.append(sid), counts.append(len(new)), ctx.append(done + len(new))
            tables.append(self.cache.block_table(sid)[0])
        out = None
        if tokens:
            slots = [self.cache.state_slot(s) for s in ids] if self.slots else None
            res = self.model.forward(ForwardBatch(tokens, positions, ids, counts, ctx, tables,
                                                  has_prefill=any(n > 1 for n in counts), state_slots=slots, logit_rows=rows))
            out = res.logits if rows else None
        for name in end:
            if name in self.live:
                self.cache.free(self.live.pop(name)[0])
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help=f"capacity of the cache in tokens; a request takes a multiple of {ROUND} of them")
    args = ap.parse_args(argv)
    dtype = {"bfloat16": DType.BF16, "float32": DType.F32}[args.dtype]
    runner = TraceRunner.from_directory(args.model, dtype, args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = runner.step(step["entries"], step.get("end", ()))
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0
