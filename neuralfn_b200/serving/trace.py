"""Replays a trace of token batches through a model and writes the logits it asks for.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object per line:

    {"step": 7, "entries": [{"id": "chat-1", "tokens": [101, 9], "want": [1]}, {"id": "chat-2", "tokens": [44]}], "end": ["chat-1"]}

An entry holds the next tokens of one request and the places among them whose logits are wanted; all entries of a step run as one
batch (``ResidentEngine.step``). A request gets a slot at its first entry and gives everything back when ``end`` names it. The wanted
logits go to ``DIR/<step>.f32`` (little-endian fp32, [wanted, vocab], in the order of the entries and their places); after every step a
line ``done <step>`` is printed. ``--max-tokens`` sizes the cache pool, ``--slots`` (default 4) the number of live requests.

The native library is built on the first call if it is missing or out of date - only the sources this model's engine needs.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path

__all__ = ["TraceReplay", "main", "EXIT_UNSUPPORTED"]

EXIT_UNSUPPORTED = 3     # the model has no engine for the requested number format


class TraceReplay:
    """Request names on top of an engine's slots."""

    def __init__(self, engine) -> None:
        if not engine.has_steps:
            raise ValueError("this model's engine has no mixed steps; a trace cannot be replayed on it")
        self.engine = engine
        self._free = list(range(engine.config.max_batch))[::-1]
        self._slot: dict[str, int] = {}

    def run(self, step: dict):
        """One step; returns the wanted logits (fp32 [wanted, vocab]) or None when nothing was wanted."""
        from .engine import StepEntry
        entries = []
        for e in step.get("entries", ()):
            name = str(e["id"])
            if name not in self._slot:
                if not self._free:
                    raise ValueError("more live requests than slots")
                self._slot[name] = self._free.pop()
                self.engine.release(self._slot[name])
            if e["tokens"]:
                entries.append(StepEntry(self._slot[name], e["tokens"], tuple(e.get("want", ()))))
        wanted = sum(len(e.want) for e in entries)
        order = [sorted(range(len(e.want)), key=lambda i, w=e.want: w[i]) for e in entries]
        logits = None
        if entries:
            ascending = [StepEntry(e.slot, e.tokens, tuple(e.want[i] for i in o)) for e, o in zip(entries, order)]
            _, rows = self.engine.step(ascending, logits=wanted > 0)
            if wanted:
                logits, base = rows.clone(), 0
                for o in order:
                    for k, i in enumerate(o):
                        logits[base + i] = rows[base + k]
                    base += len(o)
        for name in step.get("end", ()):
            slot = self._slot.pop(str(name), None)
            if slot is not None:
                self.engine.release(slot)
                self._free.append(slot)
        return logits


def main(argv=None, stdin=None, stdout=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time (rounded up to whole pages)")
    ap.add_argument("--slots", type=int, default=4, help="live requests at any time")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    stdin, stdout = stdin or sys.stdin, stdout or sys.stdout
    from .architectures import architecture_of, load_model_directory, read_model_config
    arch = architecture_of(read_model_config(a.model))
    if a.dtype not in arch.dtypes:
        print(f"trace_run: {arch.name} does not run in {a.dtype}", file=sys.stderr)
        return EXIT_UNSUPPORTED
    from ..ops import _build, _lib
    _lib.use_library(_build.ensure_component(arch.component))
    engine = load_model_directory(a.model, device=a.device, dtype=a.dtype, max_batch=a.slots, max_seq=a.max_tokens, kv_tokens=a.max_tokens)
    replay = TraceReplay(engine)
    out = Path(a.out)
    for line in stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.run(step)
        if logits is not None:
            part = out / f".{step['step']}.part"
            part.write_bytes(logits.contiguous().numpy().astype("<f4").tobytes())
            os.replace(part, out / f"{step['step']}.f32")
        print(f"done {step['step']}", file=stdout, flush=True)
    engine.close()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
