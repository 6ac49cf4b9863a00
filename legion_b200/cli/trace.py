"""``trace``: replay steps of given tokens through a model and write logits (``bin/trace_run`` calls this too).

Steps come on standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
A step in which something is wanted writes ``OUT/<step>.f32``: little-endian float32 [wanted, vocab], in the order of the
entries and of their ``want``. After every step a line ``done <step>`` is printed. The exit code is 0 when the input
ends.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

DTYPES = ("bfloat16", "float32")


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="model directory (config.json, model.safetensors)")
    ap.add_argument("--dtype", choices=DTYPES, default="bfloat16", help="bfloat16: as served; float32: everything in 32-bit")
    ap.add_argument("--out", required=True, help="directory the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")


def ensure_built(model: str) -> None:
    """Brings the extension up to date; a checkout that was never built compiles the kernels of this model only."""
    from .. import build_ext
    if build_ext.TARGET.exists():
        build_ext.build()
        return
    from ..loaders.hf_map import config_from_hf
    with open(os.path.join(model, "config.json")) as f:
        build_ext.build_core(config_from_hf(json.load(f)))


def run(a) -> int:
    import torch
    ensure_built(a.model)
    from ..engine.replay import TraceReplay, replay_engine
    torch.backends.cuda.matmul.allow_tf32 = False
    replay = TraceReplay(replay_engine(a.model, getattr(torch, a.dtype), a.max_tokens))
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = replay.step(st["entries"], st.get("end", []))
        if logits is not None:
            part = os.path.join(a.out, f".{st['step']}.part")
            with open(part, "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
            os.replace(part, os.path.join(a.out, f"{st['step']}.f32"))
        print(f"done {st['step']}", flush=True)
    replay.engine.shutdown()
    return 0


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of steps through a model and write logits")
    add_arguments(ap)
    return run(ap.parse_args(argv))
