"""Trace runner: feeds given token ids through a model step by step and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

Every entry is the next portion of a request; all entries of a step run as one mixed step of the session (the step that
continuous batching drives).  Logits at the wanted places go to DIR/<step>.f32 as little-endian f32 [wanted, vocab], in
the order of the entries and of "want"; after every step a line "done <step>" is printed.  Requests named in "end" give
their stream and pages back.  The page pool holds N positions, shared by four streams.
"""
import argparse
import json
import os
import sys

import numpy as np

STREAMS = 4
PAGE_TOKENS = 64
STEP_ROWS = 4096  # rows of one pass at most; a longer step runs as several passes


def replay(session, lines, out_dir, done):
    """Run the steps of `lines` on a session; done(step) after each."""
    free = list(range(session.n_streams - 1, -1, -1))
    stream_of = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries, order = [], []
        for e in step["entries"]:
            if not e["tokens"]:
                continue
            if e["id"] not in stream_of:
                if not free:
                    raise RuntimeError("request %s: all %d streams are taken" % (e["id"], session.n_streams))
                stream_of[e["id"]] = free.pop()
            # the session takes ascending places; a row asked for out of order or twice is put in place below
            places = sorted(set(e["want"]))
            at = sum(len(p) for _, _, p in entries)
            entries.append((stream_of[e["id"]], e["tokens"], places))
            order += [at + places.index(w) for w in e["want"]]
        if entries:
            logits = session.step(entries)
            if order:
                rows = np.ascontiguousarray(logits[order], dtype="<f4")
                part = os.path.join(out_dir, ".%s.part" % step["step"])
                rows.tofile(part)
                os.replace(part, os.path.join(out_dir, "%s.f32" % step["step"]))
        for name in step.get("end", []):
            if name in stream_of:
                s = stream_of.pop(name)
                session.reset(s)
                free.append(s)
        done(step["step"])


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of steps through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", required=True, type=int, help="positions that live requests hold at most, in whole pages of 64")
    args = ap.parse_args(argv)
    if args.max_tokens < 1:
        ap.error("--max-tokens must be positive")
    from . import build, capi
    capi.use_library(build.ensure("plain"))
    from . import registry
    from .model import Session
    ctx = capi.Ctx(0)
    pool = (args.max_tokens + PAGE_TOKENS - 1) // PAGE_TOKENS * PAGE_TOKENS
    model = registry.load(ctx, args.model, max_context=pool, compute=args.dtype)
    session = Session(ctx, model, None, STREAMS, 1, page_tokens=PAGE_TOKENS, pool_tokens=pool, step_rows=min(pool, STEP_ROWS))

    def done(step):
        print("done %s" % step, flush=True)

    replay(session, sys.stdin, args.out, done)
    session.close(), model.close(), ctx.close()
    return 0
