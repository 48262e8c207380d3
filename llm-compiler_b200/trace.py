"""Trace replay: steps of given token ids through a model's own step function, logits written to files.

A step is one JSON object on a line of the input: {"step": n, "entries": [{"id", "tokens", "want"}, ...],
"end": [ids]}. The tokens of an entry continue the sequence of that id; the logits at the wanted places
go to <out>/<step>.f32 (little-endian fp32, [wanted, vocab]); "done <step>" follows on the output."""

from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, Iterable, TextIO

from . import kernels


def replay(engine, lines: Iterable[str], out: Path, output: TextIO) -> None:
    import torch

    slots: Dict[str, int] = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries, want = [], []
        for entry in step["entries"]:
            if not entry["tokens"]:
                continue
            if entry["id"] not in slots:
                slots[entry["id"]] = engine.open()
            entries.append((slots[entry["id"]], entry["tokens"]))
            want.append(entry["want"])
        if entries:
            logits = engine.forward(entries, want)
            engine.state.check()
            if logits is not None:
                if logits.dtype != torch.float32:
                    logits = kernels.b200_contiguous(logits, torch.float32)
                (out / f"{step['step']}.f32").write_bytes(logits.cpu().contiguous().numpy().astype("<f4").tobytes())
        for name in step.get("end", []):
            if name in slots:
                engine.close(slots.pop(name))
        output.write(f"done {step['step']}\n")
        output.flush()
