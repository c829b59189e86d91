"""Replaying traces: given token ids run through a model step by step, the logits at the places asked for are written
out.  Nothing is sampled.  The steps go through the session that generation uses (session.Session.extend): portions of
a prompt through the model's prompt path, single tokens as decode steps, both on the session's caches.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

One JSON object a line on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries` bring the next tokens of requests and the places among them whose logits are wanted; `end` names requests that
are finished after the step.  OUT/<step>.f32 holds the step's logits, [wanted, vocab] little-endian fp32, in the order of
the entries; "done <step>" is printed when the step is complete.  Exit codes: 0 at the end of the input, 3 if the model
does not run in the dtype."""
from __future__ import annotations

import argparse
import json
import os
import sys


class Replay:
    """Requests by id, each on a session; the session of a finished request is reset and used again."""

    def __init__(self, model, device):
        self.model, self.device = model, device
        self.live: dict[str, object] = {}
        self.free: list = []

    def _session(self, rid: str):
        if rid not in self.live:
            from .registry import open_session
            self.live[rid] = self.free.pop() if self.free else open_session(self.model)
        return self.live[rid]

    def run(self, entry: dict):
        """The wanted logits (len(want), V) of one request's next tokens."""
        import torch
        tokens = torch.tensor([entry["tokens"]], dtype=torch.long, device=self.device)
        return self._session(entry["id"]).extend(tokens, list(entry["want"]))[0]

    def end(self, rid: str) -> None:
        sess = self.live.pop(rid, None)
        if sess is not None:
            sess.check()
            sess.reset()
            self.free.append(sess)


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", required=True, choices=("bfloat16", "float32"))
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    from . import registry
    fam = registry.family(registry.read_config(args.model))
    if args.dtype not in fam.dtypes:
        print(f"this model runs in {', '.join(fam.dtypes)} only", file=sys.stderr)
        return 3
    registry.build_for(registry.read_config(args.model))
    import torch
    if not torch.cuda.is_available():
        raise RuntimeError("nativebit_b200 needs a CUDA device")
    device = torch.device("cuda", torch.cuda.current_device())
    model = registry.load_model(args.model, args.dtype, max(1, args.max_tokens), device)
    replay = Replay(model, device)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = [replay.run(e).float().cpu() for e in step["entries"] if e["tokens"]]
        wanted = torch.cat([r for r in rows if r.shape[0]]) if any(r.shape[0] for r in rows) else None
        if wanted is not None:
            path = os.path.join(args.out, f"{step['step']}.f32")
            with open(path, "wb") as f:
                f.write(wanted.contiguous().numpy().astype("<f4", copy=False).tobytes())
        for rid in step.get("end", []):
            replay.end(rid)
        print(f"done {step['step']}", flush=True)
    return 0
