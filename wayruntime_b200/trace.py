"""Replay of a trace: given token ids go through a model step by step and the asked logits are written out.

Steps come as JSON lines {"step", "entries": [{"id", "tokens", "want"}], "end": [ids]}; the logits at the wanted
places go to DIR/<step>.f32 ([wanted, vocab] little-endian F32) and 'done <step>' follows each step.  Everything is
the serving path's own: the registry's loader, the engine's step function, its sessions.
"""
from __future__ import annotations

import json
import os

import numpy as np

from . import models
from .binding import Context
from .engine import Engine

PORTION_MAX = 2048


def replay(model_dir: str, dtype: str, out_dir: str, max_tokens: int, lines, write) -> None:
    ctx = Context(0, attn_max_seq=max(max_tokens, 64))
    model = models.load(ctx, model_dir, dtype, max_rows=min(max(max_tokens, 16), PORTION_MAX))
    engine = Engine(model)
    sessions = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [e for e in step["entries"] if e["tokens"]]
        for e in entries:
            if e["id"] not in sessions:
                sessions[e["id"]] = engine.session(max_tokens)
        rows = engine.advance([sessions[e["id"]] for e in entries], [e["tokens"] for e in entries],
                              [e["want"] for e in entries]) if entries else []
        if any(len(r) for r in rows):
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for i in step["end"]:
            if i in sessions:
                sessions.pop(i).close()
        write(f"done {step['step']}\n")
    for s in sessions.values():
        s.close()
    model.close()
    ctx.close()
