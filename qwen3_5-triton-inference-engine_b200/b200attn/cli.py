"""Command line of the engines: `python -m b200attn.cli <command>` (or bin/generate, bin/trace_run).

    generate   greedy generation for prompts of token ids through the continuous batcher
    trace      replay given token ids step by step and write logits
    info       the configuration of a model folder and what the registry makes of it
"""
from __future__ import annotations

import argparse
import importlib.util
import json
import sys
from pathlib import Path

PKG = Path(__file__).resolve().parent.parent
DTYPES = ("bfloat16", "float32")
UNSUPPORTED = 3          # exit code: the model's engine does not run in the wanted precision


def _build_for(part: str | None):
    """Compile what the model needs, if it is not there yet, and load it."""
    import b200attn

    spec = importlib.util.spec_from_file_location("b200_build", PKG / "build.py")
    build = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(build)
    b200attn.load(build.build() if part is None else build.ensure(part))


def _open(folder, dtype_name: str):
    from . import checkpoint, models
    import torch

    dtype = getattr(torch, dtype_name)
    fam = models.family(checkpoint.read_config(folder))
    if dtype not in fam.dtypes:
        print(f"{fam.name} does not run in {dtype_name}", file=sys.stderr)
        sys.exit(UNSUPPORTED)
    _build_for(fam.part)
    return models.load_model(folder, dtype, "cuda")


# ----------------------------------------------------------------------------------------------------------- generate
def generate(args) -> int:
    from .serving import ContinuousBatcher

    lines = [line for line in (sys.stdin if args.prompts == "-" else open(args.prompts)) if line.strip()]
    prompts = [json.loads(line) for line in lines]
    if not prompts:
        return 0
    model = _open(args.model, args.dtype)
    longest = max(len(p) for p in prompts) + args.max_new_tokens
    options = {"prefill_chunk": args.prefill_chunk} if args.prefill_chunk else {}
    engine = model.engine(min(args.slots, len(prompts)), longest, on_demand_pages=True, **options)
    batcher = ContinuousBatcher(engine, stop_ids=args.stop)
    rids = [batcher.submit(p, args.max_new_tokens) for p in prompts]
    batcher.step()                       # the first step runs eagerly; from here on every step is one graph replay
    if not batcher.done() and engine._warmed:
        engine.capture()
    out = batcher.run()
    for rid in rids:
        print(json.dumps(out[rid]))
    return 0


# -------------------------------------------------------------------------------------------------------------- trace
class TraceReplay:
    """Requests by name over the slots of one engine: every step's tokens go through `engine.extend`, which runs prompts
    and portions as packed prefills and single tokens as the decode step."""

    def __init__(self, engine):
        self.engine = engine
        self.slot: dict[str, int] = {}
        self.held: dict[str, int] = {}
        self.free = list(range(engine.batch))[::-1]

    def step(self, entries: list[dict]):
        """fp32 logits [wanted, vocab] of the step on the CPU, or None when nothing is wanted."""
        entries = [e for e in entries if e["tokens"]]
        if not entries:
            return None
        for e in entries:
            if e["id"] not in self.slot:
                if not self.free:
                    raise RuntimeError(f"more than {self.engine.batch} live requests")
                self.slot[e["id"]] = self.free.pop()
                self.held[e["id"]] = 0
        logits = self.engine.extend([self.slot[e["id"]] for e in entries], [self.held[e["id"]] for e in entries],
                                    [e["tokens"] for e in entries], [e["want"] for e in entries])
        for e in entries:
            self.held[e["id"]] += len(e["tokens"])
        return logits.cpu() if any(e["want"] for e in entries) else None

    def end(self, names) -> None:
        for name in names:
            slot = self.slot.pop(name, None)
            if slot is not None:
                self.engine.pages.release(slot)
                self.held.pop(name)
                self.free.append(slot)


def trace(args) -> int:
    model = _open(args.model, args.dtype)
    # every request may hold all of the tokens: a slot's table row covers max-tokens, the pool holds them once, plus the
    # part-filled page of every slot and the spare page
    engine = model.engine(args.slots, args.max_tokens, on_demand_pages=True,
                          num_pages=-(-args.max_tokens // 16) + args.slots + 1)
    replay = TraceReplay(engine)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"])
        if logits is not None:
            (out / f"{step['step']}.f32").write_bytes(logits.numpy().astype("<f4").tobytes())
        replay.end(step.get("end", []))
        print(f"done {step['step']}", flush=True)
    return 0


def info(args) -> int:
    from . import checkpoint, models

    config = checkpoint.read_config(args.model)
    fam = models.family(config)
    print(json.dumps({"architecture": fam.name, "dtypes": [str(d).removeprefix("torch.") for d in fam.dtypes],
                      "layers": [layer["type"] for layer in config.get("layers", [])]}))
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="b200attn", description=__doc__.split("\n")[0])
    sub = ap.add_subparsers(dest="command", required=True)
    p = sub.add_parser("generate", help="greedy generation through the continuous batcher")
    p.add_argument("--model", required=True)
    p.add_argument("--dtype", choices=DTYPES, default="bfloat16")
    p.add_argument("--prompts", default="-", help="file with one JSON list of token ids per line ('-': standard input)")
    p.add_argument("--max-new-tokens", type=int, default=32)
    p.add_argument("--slots", type=int, default=32, help="sequences that decode together")
    p.add_argument("--prefill-chunk", type=int, default=None, help="longest portion of a prompt run at once")
    p.add_argument("--stop", type=int, nargs="*", default=[], help="token ids that end a request")
    p.set_defaults(run=generate)
    p = sub.add_parser("trace", help="replay token ids from standard input, write logits")
    p.add_argument("--model", required=True)
    p.add_argument("--dtype", choices=DTYPES, required=True)
    p.add_argument("--out", required=True, help="folder for <step>.f32 files")
    p.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    p.add_argument("--slots", type=int, default=4, help="requests that may be live at once")
    p.set_defaults(run=trace)
    p = sub.add_parser("info", help="what the registry makes of a model folder")
    p.add_argument("--model", required=True)
    p.set_defaults(run=info)
    args = ap.parse_args(argv)
    return args.run(args)


if __name__ == "__main__":
    sys.exit(main())
