"""Command line over the engine, for any model of the registry.

``generate``: greedy continuations.  Prompts are token ids, one prompt a line on standard input (separated by
spaces or commas); the continuation's ids are printed, one line per prompt.

``trace``: replays given tokens.  Each line of standard input is one step,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` brings the next tokens of some requests and the places among them whose logits are wanted, ``end`` names
the requests that are finished after the step.  The wanted logits go to ``OUT/<step>.f32`` (little-endian floats,
[wanted, vocab], in the order of the entries), and ``done <step>`` is printed after every step.

Both compile the kernel libraries the model needs if they are missing or out of date."""
from __future__ import annotations

import argparse
import json
import os
import sys

DTYPES = ("bfloat16", "float16", "float32")
TRACE_REQUESTS = 16      # requests that can be live at once when replaying
TRACE_BLOCK = 256        # the engine's own block size: the kernels are those of serving


def _model(args):
    """(model, None), or (None, exit code) where the model does not run in the type that was asked for."""
    import torch
    from .csrc import build
    from .models import build_model, model_class, read_config
    entry = model_class(read_config(args.model))
    dtype = getattr(torch, args.dtype)
    if dtype not in entry.dtypes:
        print(f"this model does not run in {args.dtype}", file=sys.stderr)
        return None, 3
    for name in entry.libraries:
        build.build_library(getattr(build, name))
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    torch.cuda.set_device(0)
    return build_model(args.model, device="cuda:0", dtype=dtype), None


def _generate(args) -> int:
    model, code = _model(args)
    if model is None:
        return code
    from .engine import LLMEngine
    prompts = [[int(t) for t in line.replace(",", " ").split()] for line in sys.stdin if line.strip()]
    longest = max((len(p) for p in prompts), default=0) + args.max_new_tokens + 1
    blocks = args.blocks or min(args.max_batch, max(len(prompts), 1)) * -(-longest // args.block_size)
    engine = LLMEngine(model, num_blocks=blocks, block_size=args.block_size, max_batch=args.max_batch, prefill_portion=args.portion)
    for out in engine.generate(prompts, args.max_new_tokens):
        print(" ".join(map(str, out)), flush=True)
    return 0


def _trace(args) -> int:
    model, code = _model(args)
    if model is None:
        return code
    import torch
    from .engine import LLMEngine, Sequence
    blocks = -(-args.max_tokens // TRACE_BLOCK) + TRACE_REQUESTS
    engine = LLMEngine(model, num_blocks=blocks, block_size=TRACE_BLOCK, max_batch=TRACE_REQUESTS)
    live: dict[str, Sequence] = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            seq = live.get(e["id"])
            if seq is None:
                seq = live[e["id"]] = Sequence(len(live), [], 1 << 62)
            if e["tokens"]:
                entries.append((seq, e["tokens"], e.get("want") or []))
        logits = [t for t in engine.extend(entries) if t is not None] if entries else []
        if logits:
            data = torch.cat(logits).float().cpu().numpy().astype("<f4")
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as fh:
                fh.write(data.tobytes())
        for name in step.get("end") or []:
            engine.drop(live.pop(name))
        print(f"done {step['step']}", flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="nanoquantization_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy continuations of prompts of token ids")
    t = sub.add_parser("trace", help="replay given tokens and write logits")
    for p in (g, t):
        p.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
        p.add_argument("--dtype", default="bfloat16", choices=DTYPES)
    g.add_argument("--max-new-tokens", type=int, default=16)
    g.add_argument("--max-batch", type=int, default=64)
    g.add_argument("--block-size", type=int, default=256)
    g.add_argument("--blocks", type=int, default=0, help="K/V blocks (default: enough for the prompts)")
    g.add_argument("--portion", type=int, default=None, help="tokens of a prefill step at most; longer prompts run in portions")
    t.add_argument("--out", required=True, help="folder for the logits")
    t.add_argument("--max-tokens", type=int, default=65536, help="tokens that live requests hold at any time, at most")
    args = ap.parse_args(argv)
    return _generate(args) if args.command == "generate" else _trace(args)


if __name__ == "__main__":
    sys.exit(main())
