"""Command line of the framework.

    python -m kinetics_b200 generate --model DIR --prompt 5,17,3 --prompt 8,1 --max-new-tokens 32
    python -m kinetics_b200 trace    --model DIR --dtype bfloat16 --out DIR --max-tokens N      (= bin/trace_run)

`generate` takes prompts as token ids (no tokenizer is part of this package), runs them through Engine -- slots, page
pool, sampler -- and prints one JSON object per request.  `trace` replays given tokens step by step from standard
input and writes the logits asked for.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def _parse(argv):
    ap = argparse.ArgumentParser(prog="kinetics_b200")
    sub = ap.add_subparsers(dest="command", required=True)

    def common(p):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
        p.add_argument("--device", default="cuda:0")
        p.add_argument("--page-size", type=int, default=64, choices=[16, 32, 64], help="tokens per cache page")

    g = sub.add_parser("generate", help="generate from prompts of token ids")
    common(g)
    g.add_argument("--prompt", action="append", default=[], help="token ids with commas between them; repeatable")
    g.add_argument("--requests", help="file of JSON lines {\"input_ids\": [...]} (- for standard input)")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--max-batch", type=int, default=8)
    g.add_argument("--num-pages", type=int, default=0, help="pages of the cache (0: enough for every slot)")
    g.add_argument("--prefill-chunk", type=int, default=0, help="run prompts in portions of this many tokens (0: whole)")
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=None)
    g.add_argument("--eos", default="", help="token ids that end a sequence, with commas between them")

    t = sub.add_parser("trace", help="replay tokens from standard input and write logits")
    common(t)
    t.add_argument("--out", required=True, help="folder for <step>.f32")
    t.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live requests hold")
    return ap.parse_args(argv)


def _ids(text: str):
    return [int(x) for x in text.replace(",", " ").split()]


def generate(args, out=sys.stdout) -> int:
    from .engine import Engine
    from .registry import load_model

    requests = [{"input_ids": _ids(p)} for p in args.prompt]
    if args.requests:
        with (sys.stdin if args.requests == "-" else open(args.requests)) as f:
            requests += [json.loads(line) for line in f if line.strip()]
    if not requests or any(not r["input_ids"] for r in requests):
        print("generate: no prompt, or an empty one", file=sys.stderr)
        return 2
    for i, r in enumerate(requests):
        r.setdefault("id", i)
    model = load_model(args.model, args.device, DTYPES[args.dtype])
    longest = max(len(r["input_ids"]) for r in requests) + args.max_new_tokens + 1
    kv = model.new_cache(min(args.max_batch, len(requests)), longest, args.num_pages or None, args.page_size)
    engine = Engine(model, kv, longest, args.device, top_p=args.top_p, temperature=args.temperature, top_k=args.top_k,
                    eos=_ids(args.eos), repeat_check=False, seed=args.seed, prefill_chunk=args.prefill_chunk)
    for r in sorted(engine.offline_exec(requests, args.max_new_tokens), key=lambda r: str(r["id"])):
        print(json.dumps({"id": r["id"], "output_tokens": r["output_tokens"]}), file=out)
    kv.check_status()
    model.check_status()
    return 0


def trace(args, lines=None, out=sys.stdout) -> int:
    """Every input line {"step", "entries": [{"id", "tokens", "want"}], "end": [ids]} runs its entries on top of what
    earlier steps left in the requests' slots, writes OUT/<step>.f32 (the wanted logits, fp32, in order) and answers
    'done <step>'; ended requests give their slots and pages back."""
    from .engine import Engine
    from .registry import load_model

    slots = 8
    model = load_model(args.model, args.device, DTYPES[args.dtype])
    pages = (args.max_tokens + args.page_size - 1) // args.page_size + slots
    kv = model.new_cache(slots, max(args.max_tokens, 1), pages, args.page_size)
    engine = Engine(model, kv, max(args.max_tokens, 1), args.device, repeat_check=False)
    slot_of = {}
    for line in (sys.stdin if lines is None else lines):
        if not line.strip():
            continue
        step = json.loads(line)
        wanted = []
        for entry in step["entries"]:
            if entry["id"] not in slot_of:
                free = [s for s in range(slots) if not engine.slots_occupy_status[s]]
                if not free:
                    raise RuntimeError(f"more than {slots} live requests")
                slot_of[entry["id"]] = free[0]
                engine.open_slot(free[0])
            logits = engine.extend(slot_of[entry["id"]], entry["tokens"], entry["want"])
            if logits is not None:
                wanted.append(logits.float().cpu())
        kv.check_status()
        model.check_status()
        if wanted:
            torch.cat(wanted).contiguous().numpy().astype("<f4").tofile(str(Path(args.out) / f"{step['step']}.f32"))
        for name in step["end"]:
            if name in slot_of:
                engine.clear_request(slot_of.pop(name))
        print(f"done {step['step']}", file=out, flush=True)
    return 0


def main(argv=None) -> int:
    args = _parse(sys.argv[1:] if argv is None else argv)
    if args.device.startswith("cuda") and not torch.cuda.is_available():
        print("kinetics_b200: no CUDA device (there is no CPU path)", file=sys.stderr)
        return 1
    if args.device.startswith("cuda"):
        torch.cuda.set_device(args.device)
    torch.backends.cuda.matmul.allow_tf32 = False
    return generate(args) if args.command == "generate" else trace(args)
