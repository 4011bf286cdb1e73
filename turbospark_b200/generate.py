"""Generate from a model folder (config.json, model.safetensors), prompts and output as token ids.

    python -m turbospark_b200.generate --model DIR --prompt "5 17 3" --prompt "8 1" --max-new-tokens 32

Every prompt is a request; they are served together by continuous batching.  One JSON line per request.
"""
import argparse
import json
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="token ids, separated by spaces or commas; may be given several times")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--streams", type=int, default=4, help="requests that run at the same time")
    ap.add_argument("--pool-tokens", type=int, default=0, help="positions the page pool holds (0: enough for every stream)")
    ap.add_argument("--prefill-chunk", type=int, default=1024, help="prompt tokens of one request per step at most")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=0.0)
    ap.add_argument("--min-p", type=float, default=0.0)
    ap.add_argument("--repetition-penalty", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--stop", type=int, action="append", default=[], help="a token id that ends a request (up to eight)")
    args = ap.parse_args(argv)
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in args.prompt]
    if any(not p for p in prompts) or args.max_new_tokens < 1 or args.streams < 1:
        ap.error("every prompt has tokens, and --max-new-tokens and --streams are positive")

    from . import build, capi
    if capi._lib is None:
        capi.use_library(build.ensure("plain"))
    from . import registry
    from .model import Session, run_config
    ctx = capi.Ctx(0)
    context = max(len(p) for p in prompts) + args.max_new_tokens
    model = registry.load(ctx, args.model, max_context=context, compute=args.dtype)
    streams = min(args.streams, len(prompts))
    session = Session(ctx, model, None, streams, 1, pool_tokens=args.pool_tokens, step_rows=min(4096, max(context, 2 * streams)))
    rc = run_config(capi.shaping(temperature=args.temperature, top_k=args.top_k, top_p=args.top_p, min_p=args.min_p,
                                 repetition_penalty=args.repetition_penalty, seed=args.seed), args.max_new_tokens, 1, stop_tokens=args.stop[:8])
    out, reasons, stats = session.serve(prompts, [args.max_new_tokens] * len(prompts), rc, prefill_chunk=args.prefill_chunk)
    for p, t, r in zip(prompts, out, reasons):
        print(json.dumps({"prompt": p, "tokens": t.tolist(), "reason": "stop" if r else "length"}))
    print("%d requests, %d steps, %d rows, %.3f s" % (len(prompts), stats.steps, stats.rows, stats.seconds), file=sys.stderr)
    session.close(), model.close(), ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
