"""Trace replay: feed given token ids through a model step by step and write logits (the program behind bin/trace_run).

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N   < steps.jsonl

One step per input line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  `tokens` continue the request
`id`, `want` names places among them; their logits go to OUT/<step>.f32 (little-endian fp32, [wanted, vocab]) in the order of
the entries.  Requests in `end` give their slot and pages back after the step.  "done <step>" is printed after every step.
The engine, its passes, cache and kernels are the serving ones (models/registry.py); nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List

DTYPES = {"bfloat16": "bf16", "float32": "f32"}
EXIT_NO_DTYPE = 3
MAX_ROWS = 1024
SLOTS = 32


class Replay:
    def __init__(self, engine):
        self.e = engine
        self.slot: Dict[str, int] = {}
        self.at: Dict[int, int] = {}

    def step(self, entries: List[dict]):
        """Run the entries' tokens in as few passes as fit; yields the wanted logits rows in order."""
        import torch
        e = self.e
        rows, want = [], []                     # (token, position, slot) and index of every wanted row
        for en in entries:
            if en["id"] not in self.slot:
                lease = e.cache.admit()
                if lease is None:
                    raise RuntimeError("every slot is in use")
                self.slot[en["id"]] = lease[0]
                self.at[lease[0]] = 0
            slot = self.slot[en["id"]]
            pos = self.at[slot]
            n = len(en["tokens"])
            if not e.cache.ensure(slot, pos + n):
                raise RuntimeError("the cache cannot hold this step")
            want += [len(rows) + w for w in en["want"]]
            rows += [(t, pos + i, slot) for i, t in enumerate(en["tokens"])]
            self.at[slot] = pos + n
        got = {}
        for c0 in range(0, len(rows), e.max_rows):
            part = rows[c0:c0 + e.max_rows]
            e.set_rows(*[list(x) for x in zip(*part)])
            e.forward_rows(len(part), head=False)
            here = sorted({w for w in want if c0 <= w < c0 + len(part)})
            if here:
                for w, row in zip(here, e.logits_at([w - c0 for w in here])):
                    got[w] = row
        e.check_status("trace replay")
        return torch.stack([got[w] for w in want]).float().cpu() if want else None

    def end(self, rid: str):
        slot = self.slot.pop(rid, None)
        if slot is not None:
            del self.at[slot]
            self.e.cache.release(slot)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and its safetensors files")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    from ..models import registry
    dtype = DTYPES[args.dtype]
    fam, _ = registry.config_from_file(args.model)
    if dtype not in fam.dtypes:
        print(f"trace_run: {fam.name} models do not run in {args.dtype}", file=sys.stderr)
        return EXIT_NO_DTYPE
    import torch
    dev = torch.device("cuda", args.device)
    torch.cuda.set_device(dev)
    n = max(args.max_tokens, 64)
    engine = registry.load_engine(args.model, dev, dtype, max_rows=min(MAX_ROWS, n), slots=SLOTS, max_ctx=n,
                                  n_pages=-(-n // 64) + SLOTS)
    run = Replay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = run.step(step["entries"])
        if logits is not None:
            logits.numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        for rid in step.get("end", []):
            run.end(rid)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
