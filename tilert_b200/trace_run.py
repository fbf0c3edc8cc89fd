"""Replays recorded token ids: every request's tokens go through a model in the steps of the recording, and the logits
at the places a step names are written out.  Nothing is sampled.

    bin/trace_run --model MODEL_DIR --out LOGITS_DIR [--dtype float32] [--max-tokens N] < steps.jsonl

A step is one line of JSON,

    {"step": 7, "entries": [{"id": "chat-1", "tokens": [11, 12], "want": [1]}], "end": ["chat-1"]}

where ``want`` holds indices into ``tokens`` and ``end`` names requests that are over.  LOGITS_DIR/7.f32 then holds the
logits as raw little-endian f32 rows, and the line "done 7" follows.  The model runs one sequence at a time: a request
continues where its previous step ended, and another may begin once it is over.  Exit code 3: the model's family does not
run in the given type.
"""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


class TraceRunner:
    """Steps of a trace on one ``SequenceDriver``."""

    def __init__(self, model):
        self.model = model
        self.active = None  # id of the request the model's sequence belongs to

    def step(self, entries: list[dict], end: list):
        """Run a step's entries; returns the wanted logits [wanted, vocab] or None."""
        import torch

        outs = []
        for e in entries:
            if self.active is None:
                self.model.reset_sequence()
                self.active = e["id"]
            elif self.active != e["id"]:
                raise ValueError(f"request {e['id']!r} while {self.active!r} is live: the model holds one sequence")
            tokens, want = [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", [])]
            if tokens:
                outs.append(self.model.prefill(tokens, want))
        for rid in end:
            if rid != self.active:
                raise ValueError(f"request {rid!r} is not live")
            self.active = None
            self.model.reset_sequence()
        outs = [o for o in outs if o.shape[0]]
        return torch.cat(outs) if outs else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, default=None, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)

    from tilert_b200.models.registry import family_of_dir

    family = family_of_dir(a.model)
    if a.dtype not in family.dtypes:
        print(f"{family.name} runs in {', '.join(family.dtypes)}, not in {a.dtype}", file=sys.stderr)
        return 3
    from tilert_b200 import build

    build.build(model_type=family.backend)  # a fresh checkout has no libraries yet
    import tilert_b200 as tb

    model = family.load(a.model, "cuda:0", a.dtype, a.max_tokens)
    runner, out = TraceRunner(model), Path(a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step(s["entries"], s.get("end", []))
        if logits is not None:
            (out / f"{s['step']}.f32").write_bytes(logits.float().cpu().contiguous().numpy().astype("<f4").tobytes())
        status = tb.device_status(0, model.backend)
        if status != 0:
            raise RuntimeError(f"a kernel gave up with status {status}")
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
