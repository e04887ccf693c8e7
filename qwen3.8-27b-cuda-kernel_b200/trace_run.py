"""Trace replay: feeds given token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON object per line: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}.
`entries` brings each request's next tokens and the places among them whose logits are wanted, `end` the requests that
are finished after the step. For a step with wanted places DIR/<step>.f32 receives them as little-endian fp32
[wanted][vocab]; after every step a line `done <step>` is printed. Nothing is sampled.

Everything runs through ModelRunner: several tokens of a request are a prefill step (in chunks), a single token is a
decode step, pages and slots come from the runner's cache and are given back at the end of a request.
"""

from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path

REFUSED = 3


def _libraries(model_dir: Path) -> None:
    """Builds what this model's family needs, unless the full build is already there."""
    import q38b200

    from . import build as builder
    try:
        name = json.loads((model_dir / "config.json").read_text())["architecture"]
    except (OSError, KeyError, ValueError):
        name = None
    family = builder.ARCHITECTURE_FAMILY.get(name)
    full = builder.up_to_date(None)
    libs = builder.build(family=None if full else family)
    q38b200.use_libraries(libs["engine"].parent)


class Replay:
    """Requests by name on the runner's slots."""

    def __init__(self, eng, model, runner, options):
        self.eng, self.model, self.runner = eng, model, runner
        self.chunk = options.prefill_chunk
        self.free = list(range(options.max_batch))[::-1]
        self.slot: dict[str, int] = {}
        self.held: dict[str, int] = {}

    def _enter(self, name: str, new: int) -> None:
        if name not in self.slot:
            if not self.free:
                raise SystemExit(f"trace_run: more than {len(self.slot)} live requests")
            self.slot[name], self.held[name] = self.free.pop(), 0
            self.runner.reset_slot(self.slot[name])
        if not self.runner.kv_ensure(self.slot[name], self.held[name] + new):
            raise SystemExit("trace_run: the cache is full (raise --max-tokens)")

    def _decode(self, batch):
        greedy = self.eng.greedy()
        self.runner.decode([(self.slot[n], self.held[n], t[0], greedy, 0) for n, t in batch])
        return self.runner.last_logits(len(batch))

    def step(self, entries):
        """Logits of all wanted places, in the order of the entries and of their `want`."""
        import numpy as np

        entries = [e for e in entries if e["tokens"]]
        for e in entries:
            self._enter(e["id"], len(e["tokens"]))
        got = [[None] * len(e["want"]) for e in entries]
        if entries and all(len(e["tokens"]) == 1 for e in entries):
            logits = self._decode([(e["id"], e["tokens"]) for e in entries])
            for i, e in enumerate(entries):
                got[i] = [logits[i]] * len(e["want"])
                self.held[e["id"]] += 1
        else:
            at = [0] * len(entries)
            while True:  # ragged steps of at most one chunk of tokens
                rows, who, budget = [], [], self.chunk
                for i, e in enumerate(entries):
                    n = min(budget, len(e["tokens"]) - at[i])
                    if n <= 0:
                        continue
                    rows.append((self.slot[e["id"]], self.held[e["id"]], e["tokens"][at[i]:at[i] + n], None, 0))
                    who.append((i, at[i], n))
                    budget -= n
                if not rows:
                    break
                want, place = [], []
                for r, (i, lo, n) in enumerate(who):
                    for k, p in enumerate(entries[i]["want"]):
                        if lo <= p < lo + n:
                            want.append((r, p - lo))
                            place.append((i, k))
                if want:
                    logits = self.runner.step_logits(rows, want)
                    for j, (i, k) in enumerate(place):
                        got[i][k] = logits[j]
                else:
                    self.runner.prefill(rows)
                for i, lo, n in who:
                    at[i] = lo + n
                    self.held[entries[i]["id"]] += n
        flat = [row for rows in got for row in rows]
        return np.stack(flat) if flat else None

    def end(self, name: str) -> None:
        if name in self.slot:
            self.runner.kv_release(self.slot[name])
            self.free.append(self.slot.pop(name))
            del self.held[name]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="Replay a trace of token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=8, help="most live requests")
    a = ap.parse_args(argv)
    _libraries(Path(a.model))
    from . import engine as eng

    model = eng.Model(a.model)
    options = eng.default_runner_options(
        max_batch=a.slots, prefill_chunk=1024, kv_tokens=a.max_tokens + 64 * a.slots, kv_dtype=-1, verbose=0,
        max_context=max(64, min(model.max_positions, a.max_tokens)), compute_dtype=eng.COMPUTE_F32 if a.dtype == "float32" else eng.COMPUTE_BF16)
    try:
        runner = eng.Runner(model, options)
    except eng.EngineError as e:
        if a.dtype == "float32" and "bfloat16 only" in str(e):
            print(f"trace_run: {e}", file=sys.stderr)
            return REFUSED
        raise
    replay = Replay(eng, model, runner, options)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"])
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for name in step.get("end", []):
            replay.end(name)
        print(f"done {step['step']}", flush=True)
    runner.close()
    model.close()
    return 0
