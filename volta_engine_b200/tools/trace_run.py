"""``trace_run``: feed given token ids through a model step by step and write logits. Nothing is sampled.

  trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line on standard input is one step, one batch of the engine:

  {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries``: the next tokens of each request and the places among them whose logits are wanted; ``end``: requests that are
finished after the step. A request is admitted at its first entry (it takes a state slot and, as it grows, cache pages) and
gives them back at its end. The logits go to ``OUT/<step>.f32`` (little-endian fp32 [wanted, vocab], in the order of the
entries and places); after every step the line ``done <step>`` is printed. The engine is the one the server builds
(``build_engine``): cache pool of ``--max-tokens`` tokens, ``--slots`` state slots, decode steps as graph replays.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


class TraceRunner:
    """Requests by name on an engine: slots, positions, one forward per step."""

    def __init__(self, engine):
        self.engine = engine
        self.free = list(range(engine.kv.max_slots - 1, -1, -1))
        self.live: dict[str, list] = {}                    # id -> [slot, tokens so far]

    def step(self, entries: list, end: list):
        """-> wanted logits (fp32 [wanted, vocab]) or None."""
        segs = []
        for e in entries:
            toks = [int(t) for t in e["tokens"]]
            if not toks:
                continue
            r = self.live.get(e["id"])
            if r is None:
                if not self.free:
                    raise RuntimeError(f"request {e['id']!r}: all {self.engine.kv.max_slots} slots are taken")
                r = self.live[e["id"]] = [self.free.pop(), 0]
            segs.append((r[0], toks, r[1], [int(w) for w in e.get("want", [])]))
            r[1] += len(toks)
        logits = self.engine.forward_segments(segs) if segs else None
        if logits is not None:
            logits = logits.float().cpu()
        for name in end:
            r = self.live.pop(name, None)
            if r is not None:
                self.engine.kv.release(r[0])
                self.free.append(r[0])
        return logits


def build(model_dir: str, dtype: str, max_tokens: int, slots: int, device=None):
    import torch
    from .. import _lib
    from ..models.factory import kernel_sources
    from ..server.cli import build_engine, resolve_config
    part = kernel_sources(model_dir)
    if part is not None and torch.cuda.is_available() and device != "cpu":
        _lib.kernels_of(*part)                             # in a fresh checkout: compile what this model needs
    n = (max_tokens + 63) // 64 * 64
    cfg, _ = resolve_config(["--model-dir", model_dir, "--set", f"dtype={'fp32' if dtype == 'float32' else 'bf16'}", "--set", f"kv_pool={n}",
                             "--set", f"max_seq={n}", "--set", f"max_slots={slots}", "--set", "scratch_mib=64"], env={})
    _, _, engine, _ = build_engine(cfg, device)
    return engine


def main(argv=None, stdin=None, device=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder that receives <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=4, help="most requests that are live at any time")
    a = ap.parse_args(argv)
    try:
        engine = build(a.model, a.dtype, a.max_tokens, a.slots, device)
    except NotImplementedError as ex:
        print(f"trace_run: {ex}", file=sys.stderr)
        return 3 if a.dtype == "float32" else 2
    if not engine.supports_mixed:
        print(f"trace_run: {type(engine.model).__name__} does not take mixed batches", file=sys.stderr)
        return 2
    runner = TraceRunner(engine)
    for line in (stdin or sys.stdin):
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step(s.get("entries", []), s.get("end", []))
        if logits is not None:
            with open(os.path.join(a.out, f"{s['step']}.f32"), "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4", copy=False).tobytes())
        print(f"done {s['step']}", flush=True)
    if engine.cuda:
        from ..ops import kernels as K
        if K.check_status(engine.device):
            print("trace_run: a device-side wait ran out", file=sys.stderr)
            return 1
    return 0


if __name__ == "__main__":
    sys.exit(main())
