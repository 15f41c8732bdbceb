"""Replays a trace of given tokens through the engine and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Standard input holds one JSON object per line,

    {"step": 7, "entries": [{"id": "left", "tokens": [11, 4], "want": [1]}], "end": ["left"]}

with the next tokens of some requests, the indexes (within these tokens) whose logits are to be
kept, and the requests that give back their cache and state once the step is through.  A step that
keeps any leaves DIR/<step>.f32 (little-endian float32, one vocabulary row each, entry by entry);
"done <step>" on standard output answers every step.  Nothing is sampled: the tokens go through
DecodeEngine.extend, the forward pass that generation uses."""
from __future__ import annotations

import argparse
import json
import os
import sys

DTYPES = {"float32": "float32", "bfloat16": "bfloat16", "float16": "float16"}
MAX_SEQS, BLOCK = 16, 16


class Replayer:
    def __init__(self, model_dir: str, dtype: str, max_tokens: int, device: str = "cuda"):
        import torch

        from . import build
        build.build_library()
        from . import loader, registry
        from .engine import DecodeEngine, Sequence
        self.torch, self.Sequence = torch, Sequence
        want = getattr(torch, DTYPES[dtype])
        if want not in registry.lookup(loader.read_config(model_dir)).dtypes:
            raise NotImplementedError(f"this model does not run in {dtype}")
        cfg, model = registry.load_model(model_dir, device=device, dtype=want)
        window = getattr(model, "window", None)
        if window is not None:                  # room for every request's ring, which is opened at its full size
            self.open_tokens = max(1, max_tokens)
            blocks = -(-min(self.open_tokens, window) // BLOCK) * MAX_SEQS
        else:                                   # room for max_tokens in all; requests take blocks as they grow
            self.open_tokens = 0
            blocks = -(-max(1, max_tokens) // BLOCK) + MAX_SEQS
        self.engine = DecodeEngine(cfg, None, MAX_SEQS, max(1, blocks), BLOCK, device=device, model=model)
        self.live, self.opened = {}, 0

    def step(self, entries: list):
        """Runs one step; returns the wanted logits on the host or None."""
        eng, torch = self.engine, self.torch
        work, rows, base = [], [], 0
        for e in entries:
            seq = self.live.get(e["id"])
            if seq is None:
                seq = self.live[e["id"]] = self.Sequence(self.opened, 0, 0, self.open_tokens)
                self.opened += 1
                if not eng.admit([seq]):
                    raise RuntimeError("the cache has no room for another request")
            work.append((seq, e["tokens"]))
            rows += [base + w for w in e["want"]]
            base += len(e["tokens"])
        hidden = eng.extend(work)
        if not rows:
            torch.cuda.synchronize()
            return None
        with torch.inference_mode():
            return eng.model.logits(hidden[torch.tensor(rows, device=hidden.device)]).float().cpu()

    def end(self, ids: list) -> None:
        for i in ids:
            self.engine.retire(self.live.pop(i))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given tokens through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="tokens that live requests hold at most")
    args = ap.parse_args(argv)
    try:
        rep = Replayer(args.model, args.dtype, args.max_tokens)
    except NotImplementedError as e:
        print(e, file=sys.stderr)
        return 3
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = rep.step(step["entries"])
        if logits is not None:
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as fh:
                fh.write(logits.numpy().astype("<f4").tobytes())
        rep.end(step.get("end", []))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
