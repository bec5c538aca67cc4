"""Trace runner: feeds given token ids through a model step by step and writes the logits that are asked for.

Steps come as JSON objects, one a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  An entry appends
its tokens to the request `id` (a new id takes a free sequence of the session); `want` are places among these tokens; a
step's wanted logits go to <out>/<step>.f32 as little-endian float32 [wanted, vocab].  Requests in `end` give their blocks
and their sequence back.  The model, its paged pool and its batches are those of the engine (executor.Session)."""
from __future__ import annotations

import argparse
import json
import os
import sys


class TraceRunner:
    def __init__(self, session, out: str):
        self.s, self.out = session, out
        self.free = list(range(session.n_seq))[::-1]
        self.slot = {}

    def step(self, job: dict) -> None:
        groups, want = [], []
        for e in job["entries"]:
            if e["id"] not in self.slot:
                if not self.free:
                    raise RuntimeError(f"more than {self.s.n_seq} live requests")
                self.slot[e["id"]] = self.free.pop()
            if e["tokens"]:
                groups.append((self.slot[e["id"]], e["tokens"]))
                want.append(e["want"])
        logits = self.s.forward(groups, want)
        if len(logits):
            logits.astype("<f4").tofile(os.path.join(self.out, f"{job['step']}.f32"))
        for i in job["end"]:
            if i in self.slot:
                q = self.slot.pop(i)
                self.s.seq_reset(q)
                self.free.append(q)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replays a trace of token ids and writes logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a GGUF file")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"],
                    help="bfloat16: the kernels that serve the model; float32: f32 arithmetic throughout")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=64, help="most live requests")
    a = ap.parse_args(argv)
    from . import build
    build.ensure()
    from . import Executor, models
    from .executor import PATH_AUTO, PATH_MMA
    block = min(16, a.max_tokens)
    with Executor(0) as ex:
        ex.set_path(PATH_AUTO if a.dtype == "bfloat16" else PATH_MMA)
        # every live request may leave one block partly filled
        s = models.load(ex, a.model, n_ctx=a.max_tokens, n_seq=a.max_requests, kv_blocks=-(-a.max_tokens // block) + a.max_requests, block_tokens=block)
        runner = TraceRunner(s, a.out)
        for line in sys.stdin:
            if line.strip():
                job = json.loads(line)
                runner.step(job)
                print(f"done {job['step']}", flush=True)
        s.free()
    return 0
