"""Trace replay: given token ids go through a model step by step and the logits of chosen positions are written out - what the engine
computes, without sampling, for comparing schedules, builds and number formats.

    cuteafd trace --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

One JSON object a line: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}.  The entries of a step run
as one batch through the serving runner (`serving.runner.EngineRunner`: the packed step, CUDA-graph replay for decode-shaped steps, the
paged cache); `want` are places among the entry's tokens, `end` the requests whose pages are given back afterwards.  For a step that wants
something OUT/<step>.f32 receives the rows [wanted, vocab] as little-endian fp32; every step is answered with the line `done <step>`.
The page pool holds `--max-tokens` tokens (whole pages of 64), and up to four requests are live at a time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path

MAX_LIVE = 4


class TraceReplay:
    def __init__(self, model: str, *, dtype: str = "bfloat16", max_tokens: int, max_live: int = MAX_LIVE, device: int = 0):
        import torch
        from ..engine.kv import PAGE, PagePool
        from ..engine.registry import build_engine, load_weights, model_spec
        from .runner import EngineRunner, attach_pool
        self.spec = model_spec(model, dtype=dtype)
        dev = torch.device("cuda", device)
        torch.cuda.set_device(dev)
        pages = -(-max_tokens // PAGE) + 1                      # page 0 is the pool's scratch page
        self.engine = build_engine(self.spec, load_weights(model, self.spec, dev), n_pages=pages, max_seqs=max_live, max_pages_per_seq=pages)
        self.pool = PagePool(pages)
        self.runner = attach_pool(EngineRunner(self.engine, max_rows=16384), self.pool)
        self.live: dict = {}

    def step(self, entries: list, end: list):
        """Runs one step; returns the wanted logit rows (fp32 [wanted, vocab] on the host) or None."""
        from ..engine.kv import SeqKV
        from .scheduler import Request, Row, SeqState
        rows = []
        for e in entries:
            if not e["tokens"]:
                continue
            st = self.live.get(e["id"])
            if st is None:
                st = self.live[e["id"]] = SeqState(Request(e["id"], []), SeqKV())
            rows.append(Row(st, list(e["tokens"]), st.seq.length, list(e.get("want", []))))
        out = None
        if rows:
            self.runner.run(rows)
            commit = getattr(self.runner, "commit", None)
            if commit is not None:
                commit([(r.state, len(r.tokens)) for r in rows])        # every token given is kept
            for r in rows:
                r.state.req.prompt += r.tokens
                r.state.seq.length += len(r.tokens)
            n = sum(len(r.want_logits) for r in rows)
            if n:
                out = self.runner.last_lane.logits[:n].float().cpu()
        for rid in end:
            st = self.live.pop(rid, None)
            if st is not None:
                st.seq.release(self.pool)
                self.runner.forget(st)
        return out


def ensure_kernels(model: str):
    """A fresh checkout has no native library: build what this model's family launches, nothing else."""
    if os.environ.get("CUTEAFD_LIB"):
        return
    from .. import build
    from ..config import spec_from_snapshot
    stack = spec_from_snapshot(model).stack
    os.environ["CUTEAFD_LIB"] = str(build.ensure(f"{stack}_stack" if stack else None))


def add_arguments(ap):
    ap.add_argument("--model", required=True, help="snapshot directory")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory of the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens all live requests hold at most, each rounded up to whole pages")
    ap.add_argument("--device", type=int, default=0)


def run(a, lines=None) -> int:
    ensure_kernels(a.model)
    replay = TraceReplay(a.model, dtype=a.dtype, max_tokens=a.max_tokens, device=a.device)
    out = Path(a.out)
    for line in (sys.stdin if lines is None else lines):
        if not line.strip():
            continue
        s = json.loads(line)
        got = replay.step(s["entries"], s.get("end", []))
        if got is not None:
            (out / f"{s['step']}.f32").write_bytes(got.numpy().astype("<f4").tobytes())
        print(f"done {s['step']}", flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="replay a trace of token ids and write logits")
    add_arguments(ap)
    return run(ap.parse_args(argv))
