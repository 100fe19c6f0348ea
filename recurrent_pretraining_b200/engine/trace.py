"""Replay of a recorded request trace: token ids in, logits out, through the serving engine's own steps.

Each input line is a JSON object ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``: the next tokens of
some sequences as one batch, the places whose logits are wanted, and the sequences that are finished after the step.
Wanted logits go to ``<out>/<n>.f32`` (little-endian fp32, [wanted, vocab]); ``done <n>`` is printed after every step."""
from __future__ import annotations

import json
import os
import sys


class TraceSession:
    def __init__(self, engine):
        self.engine = engine
        self.rows: dict = {}

    def run(self, request: dict):
        """One step -> logits [wanted, vocab] or None."""
        entries = request["entries"]
        for e in entries:
            if e["id"] not in self.rows:
                self.rows[e["id"]] = self.engine.open()
        logits = None
        if entries:
            logits = self.engine.step([(self.rows[e["id"]], e["tokens"]) for e in entries], [e["want"] for e in entries])
        for i in request.get("end", []):
            self.engine.close(self.rows.pop(i))
        return logits


def replay(engine, lines, out_dir: str, answer=sys.stdout) -> None:
    session = TraceSession(engine)
    for line in lines:
        if not line.strip():
            continue
        request = json.loads(line)
        logits = session.run(request)
        n = request["step"]
        if logits is not None:
            with open(os.path.join(out_dir, f"{n}.f32"), "wb") as f:
                f.write(logits.float().cpu().contiguous().numpy().astype("<f4").tobytes())
        print(f"done {n}", file=answer, flush=True)
