"""Replay of token traces through a serving engine: the caller's tokens instead of sampled ones (``bin/trace_run``)."""
from __future__ import annotations

import json
import os
from typing import Any, Iterable, TextIO

import torch


def replay(engine: Any, lines: Iterable[str], out_dir: str, report: TextIO) -> None:
    """Runs the steps of ``lines`` (one JSON object each) and writes the wanted logits to ``out_dir/<step>.f32``."""
    live: dict[str, Any] = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open()
            entries.append((live[e["id"]], [int(t) for t in e["tokens"]], [int(p) for p in e["want"]]))
        logits = engine.feed(entries) if entries else []
        if any(e[2] for e in entries):
            data = torch.cat([t for t in logits if t.shape[0]]).float().contiguous().numpy().astype("<f4").tobytes()
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as fh:
                fh.write(data)
        for name in step["end"]:
            if name in live:
                engine.close(live.pop(name))
        report.write(f"done {step['step']}\n")
        report.flush()
    if hasattr(engine.ops, "check_status"):
        engine.ops.check_status()
