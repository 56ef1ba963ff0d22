"""Replays a trace: token ids go through a model step by step, and the logits at chosen places are written out.

One JSON object a line on standard input, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: an entry brings
the next tokens of a request and names the places among them whose logits are wanted; requests named in "end" are over and
give their slot back.  A step's logits go to OUT/<n>.f32, little-endian fp32 rows in the order of the entries and of their
"want"; after every step a line "done <n>" is printed."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Optional

import numpy as np
import torch


class TraceSession:
    """Requests of a trace by name, each in a slot of the model's caches and states."""

    def __init__(self, model, max_requests: int, max_tokens: Optional[int] = None):
        self.model = model
        model.allocate(max_requests, max_tokens)
        self.slot_of = {}

    def run(self, entries) -> np.ndarray:
        """The wanted logits of all entries, (wanted, vocab) fp32."""
        parts = []
        for e in entries:
            ids = torch.tensor([e["tokens"]], dtype=torch.int32, device="cuda")
            want = torch.tensor(e["want"], dtype=torch.int64, device="cuda")
            if not len(e["tokens"]) or any(not 0 <= w < len(e["tokens"]) for w in e["want"]):
                raise ValueError(f"request {e['id']}: empty portion, or a wanted place outside it")
            if e["id"] not in self.slot_of:
                self.slot_of[e["id"]] = self.model.slots.acquire()
            parts.append(self.model.extend(ids, [self.slot_of[e["id"]]], want).float())
        return torch.cat(parts).cpu().numpy() if parts else np.zeros((0, 0), dtype=np.float32)

    def end(self, request) -> None:
        slot = self.slot_of.pop(request, None)
        if slot is not None:
            self.model.slots.release(slot)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder that receives <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=8, help="most requests that are live at any time")
    a = ap.parse_args(argv)
    from . import registry
    try:
        model = registry.load_model(a.model, a.dtype)
    except registry.UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    if not hasattr(model, "extend"):
        print("this model family takes whole prompts only", file=sys.stderr)
        return 2
    session = TraceSession(model, a.max_requests, a.max_tokens or None)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = session.run(step["entries"])
        if logits.shape[0]:
            logits.astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for request in step.get("end", []):
            session.end(request)
        model.status()
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
