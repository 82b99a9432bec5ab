"""Replay of given tokens: feeds the token ids of a trace through a model step by step and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Standard input holds one JSON object a line,

    {"step": 0, "entries": [{"id": "a", "tokens": [811, 40, 9, 40], "want": [1, 3]}], "end": []}

``entries``: for each request its next tokens and the places among them whose logits are wanted; ``end``: requests that
are finished after the step.  Logits go to ``<out>/<step>.f32`` (little-endian fp32, [wanted, vocab], in the order of the
entries); a line ``done <step>`` follows each step.  Nothing is sampled: the steps are the serving engine's own
(:meth:`LayerEngine.step`), so a trace replays what a server would have computed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

import numpy as np


def _parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed the tokens of a trace through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=2048, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=2, help="requests that may be open at the same time")
    return ap


def run(eng, lines, out_dir: str, say) -> None:
    """Drive ``eng.step`` with the steps in ``lines``; ``say`` prints one line."""
    for line in lines:
        line = line.strip()
        if not line:
            continue
        st = json.loads(line)
        rows = []
        for e in st.get("entries", []):
            lg = eng.step(e["id"], e["tokens"], e.get("want", []))
            if lg is not None:
                rows.append(lg.cpu().numpy())
        eng.check("step %s" % st["step"])
        if rows:
            path = os.path.join(out_dir, "%d.f32" % int(st["step"]))
            np.ascontiguousarray(np.concatenate(rows, 0), dtype="<f4").tofile(path)
        for key in st.get("end", []):
            eng.end(key)
        say("done %s" % st["step"])


def main(argv: Optional[List[str]] = None) -> int:
    a = _parser().parse_args(argv)
    from .. import build as B
    from ..ops import _lib
    from ..inference import model_io as IO
    m = IO.load_model(a.model)
    _lib.use(B.ensure_layers({s.mixer.kind for s in m.cfg.layers}))
    n = max(1, a.max_tokens)
    eng = IO.build_engine(m, batch=max(1, a.slots), max_len=n, fmt={"bfloat16": "bf16", "float32": "f32"}[a.dtype])
    os.makedirs(a.out, exist_ok=True)
    run(eng, iter(sys.stdin.readline, ""), a.out, lambda s: print(s, flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
