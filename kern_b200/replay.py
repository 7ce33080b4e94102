"""Replay a trace: feed given token ids through a model, step by step, and write the logits that each step asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of standard input is one step, a batch the engine runs together:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

A request is admitted at its first entry, may sit out steps, and gives back its pages and slot after the step whose `end`
names it. A step that wants something writes `<out>/<step>.f32`: little-endian f32 [wanted, vocab], entry by entry. After
every step the line `done <step>` goes to standard output. `--max-tokens` sizes the paged pool: the most positions that
live requests hold, each rounded up to whole pages; there are state slots for `--slots` requests. Nothing is sampled: the
engine's own step runs each call, and its `logits` program reads the rows out. Exit code 3: no model here runs in the
asked-for number format.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

DTYPES = {"bfloat16": "bf16", "float32": "f32"}
ROWS = 8192             # rows of the largest call


def open_engine(model, dtype: str, max_tokens: int, slots: int = 4, cpu: bool = False):
    """An engine over a checkpoint folder whose pool holds `max_tokens` positions and `slots` requests."""
    from .engine import Engine
    from .models import registry

    page = 64
    tokens = max(page, -(-max_tokens // page) * page)
    cfg, build = registry.from_folder(model, dtype=DTYPES[dtype], page_size=page, max_tokens=min(ROWS, tokens), max_seqs=max(4, slots), max_context=tokens)
    doc = build(cfg)
    stateful = any(s.get("bytes_per_seq") for s in doc["states"].values())
    if cpu:
        from .cpu import CpuRuntime

        weights = {}
        from .models.common import read_safetensors

        for f in sorted(Path(model).glob("*.safetensors")):
            weights.update(read_safetensors(f))
        rt = CpuRuntime(doc, weights=weights, tokens=tokens, slots=slots if stateful else 0)
    else:
        from .runtime import Runtime

        rt = Runtime(doc, weights=model, tokens=tokens, slots=slots if stateful else 0)
    rt.once()
    return Engine(rt)


class Replay:
    """The live requests of a trace over one engine."""

    def __init__(self, engine):
        self.engine, self.live = engine, {}

    def step(self, entries: list[dict], end: list[str] = ()):
        """-> logits [wanted, vocab] of the step's wanted places, in order."""
        batch = []
        for e in entries:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open(len(e["tokens"]))
            batch.append((self.live[e["id"]], list(e["tokens"])))
        out = self.engine.feed(batch, [list(e.get("want", [])) for e in entries])
        self.engine.rt.check_error()
        for i in end:
            self.engine.close(self.live.pop(i))
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True)
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--slots", type=int, default=4)
    ap.add_argument("--cpu", action="store_true", help="the host-memory executor (no GPU)")
    a = ap.parse_args(argv)
    if a.dtype not in DTYPES:
        print(f"trace_run: no model runs in {a.dtype}", file=sys.stderr)
        return 3
    out = Path(a.out)
    out.mkdir(parents=True, exist_ok=True)
    run = Replay(open_engine(a.model, a.dtype, a.max_tokens, a.slots, a.cpu))
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        got = run.step(s["entries"], s.get("end", []))
        if got.shape[0]:
            (out / f"{s['step']}.f32").write_bytes(got.astype("<f4").tobytes())
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
