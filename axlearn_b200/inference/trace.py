"""Replaying a trace: given token ids go through a model in given steps, chosen logits come out.

Nothing is sampled.  The trace drives the engine that generation uses (``ModuleDecodeEngine``: prompts
through ``prefill``, single tokens through the captured step, longer continuations through ``extend``), so
a replay shows what serving computes.  Standard input has one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries``: each request's next tokens and the places among them whose logits are wanted.  ``end``:
requests that are finished after the step.  A step in which something is wanted writes ``<out>/<step>.f32``
(fp32, little-endian, ``[wanted, vocab]`` in the order of entries and wants).  After every step the line
``done <step>`` is printed.

The entries of a step are one batch.  A step either starts new requests (all from their first token; the
previous batch must have ended) or continues the current batch; requests of the batch that are not in a
step keep their states.
"""

from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Optional, Sequence

import torch

from axlearn_b200.inference.decode_engine import ModuleDecodeEngine
from axlearn_b200.inference.model_loader import LoadedModel, load_model

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class TraceReplay:
    """One batch of requests at a time on one engine."""

    def __init__(self, loaded: LoadedModel, *, max_tokens: int, device):
        self._loaded, self._max_tokens, self._device = loaded, max_tokens, torch.device(device)
        self._engine: Optional[ModuleDecodeEngine] = None
        self._rows: dict = {}        # live request id -> row of the engine's batch

    def _start(self, entries: Sequence[dict]) -> torch.Tensor:
        if self._rows:
            raise ValueError(f"new requests while {sorted(self._rows)} are still live")
        lengths = [len(e["tokens"]) for e in entries]
        ids = torch.zeros((len(entries), max(lengths)), dtype=torch.int64)
        for row, e in enumerate(entries):
            ids[row, :lengths[row]] = torch.tensor(e["tokens"])
            self._rows[e["id"]] = row
        self._engine = None          # its buffers are freed before the next batch's are allocated
        self._engine = ModuleDecodeEngine(
            self._loaded.decoder, self._loaded.parameters["decoder"], batch=len(entries),
            max_len=max(self._max_tokens, max(lengths)), dtype=self._loaded.dtype, device=self._device)
        rows = [(row, w) for row, e in enumerate(entries) for w in e["want"]]
        at = torch.tensor(rows, dtype=torch.int64).reshape(-1, 2)
        return self._engine.prefill(ids, lengths=torch.tensor(lengths), logits_at=(at[:, 0], at[:, 1]))

    def _continue(self, entries: Sequence[dict]) -> torch.Tensor:
        engine = self._engine
        steps = max(len(e["tokens"]) for e in entries)
        ids = torch.zeros((engine.batch, steps), dtype=torch.int64)
        live = torch.zeros(engine.batch, dtype=torch.int32)
        for e in entries:
            row = self._rows[e["id"]]
            ids[row, :len(e["tokens"])] = torch.tensor(e["tokens"])
            live[row] = len(e["tokens"])
        if steps == 1:
            engine.set_active(live)
            logits = engine.step_logits(ids[:, 0])[:, None]
        else:
            logits = engine.extend(ids, live)
        rows = [(self._rows[e["id"]], w) for e in entries for w in e["want"]]
        at = torch.tensor(rows, dtype=torch.int64, device=self._device).reshape(-1, 2)
        return logits[at[:, 0], at[:, 1]]

    def step(self, entries: Sequence[dict], end: Sequence[str]) -> torch.Tensor:
        """Logits ``[wanted, vocab]``."""
        entries = [e for e in entries if e["tokens"]]
        known = [e["id"] in self._rows for e in entries]
        if not entries:
            out = torch.zeros((0, 0))
        elif all(known):
            out = self._continue(entries)
        elif not any(known):
            out = self._start(entries)
        else:
            raise ValueError("a step starts requests or continues them, not both")
        for name in end:
            self._rows.pop(name, None)
        return out


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays token ids through a model; writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cpu runs the plain PyTorch statements of the operations")
    args = ap.parse_args(argv)

    # float32 means true 32-bit products.
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    torch.set_float32_matmul_precision("highest")
    if args.device != "cpu" and not torch.cuda.is_available():
        raise RuntimeError("no CUDA device")
    loaded = load_model(args.model, dtype=DTYPES[args.dtype], device=args.device)
    replay = TraceReplay(loaded, max_tokens=args.max_tokens, device=args.device)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if any(e["want"] for e in step["entries"]):
            data = logits.to(device="cpu", dtype=torch.float32).contiguous().numpy().astype("<f4").tobytes()
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        elif args.device != "cpu":
            torch.cuda.synchronize()
        print(f"done {step['step']}", flush=True)
    return 0
