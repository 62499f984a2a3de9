"""Replay of a trace: given token ids go through a model step by step, and logits come out at the places asked for.

Steps are JSON lines, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}. An entry's tokens continue what its
request has in a slot's caches and states (StepDecoder.feed: what generation runs for a prompt's portion or a new token);
an ended request gives its slot back. A step in which something is wanted writes <out>/<step>.f32, little-endian fp32 rows in
the order of the entries; every step is answered by a line "done <step>"."""

import json
from collections.abc import Iterable
from pathlib import Path
from typing import IO

from .decoder import StepDecoder


class TraceRunner:
    def __init__(self, decoder: StepDecoder):
        self.decoder = decoder
        self.free = list(range(decoder.n_slots))[::-1]
        self.live: dict[str, tuple[int, int]] = {}  # request -> (slot, positions run)

    def step(self, entries: list[dict], end: list[str]):
        """Run one step; the wanted logits as an fp32 array [wanted, vocab], or None."""
        import numpy as np

        rows = []
        for entry in entries:
            name, tokens, want = entry["id"], entry["tokens"], entry.get("want") or []
            if name not in self.live:
                if not self.free:
                    raise RuntimeError(f"more than {self.decoder.n_slots} live requests")
                self.live[name] = (self.free.pop(), 0)
            slot, done = self.live[name]
            if not tokens:
                continue
            logits = self.decoder.feed(slot, tokens, done, want)
            if want:
                rows.append(logits.cpu().numpy())
            self.live[name] = (slot, done + len(tokens))
        code = int(self.decoder.status.item())
        if code:
            raise RuntimeError(f"device status {code:#x} (NCB_DEV_* bits)")
        for name in end:
            if name in self.live:
                self.free.append(self.live.pop(name)[0])
        return np.concatenate(rows) if rows else None


def replay(decoder: StepDecoder, lines: Iterable[str], out: "str | Path", answers: IO[str]) -> None:
    runner, out = TraceRunner(decoder), Path(out)
    out.mkdir(parents=True, exist_ok=True)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = runner.step(step["entries"], step.get("end") or [])
        if logits is not None:
            logits.astype("<f4").tofile(out / f"{step['step']}.f32")
        print(f"done {step['step']}", file=answers, flush=True)
