"""Replays a trace of steps: given tokens go through an engine's own batch, cache, state and step functions.

A trace step names, per request, the tokens that come next and the places among them whose logits are wanted; all
requests of a step run as one batch. Nothing is sampled. A request is admitted at its first entry (``LmEngine.open_sequence``)
and gives its blocks and state slot back when the trace ends it, so later requests run in pages and slots that were
used before.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .lm import EngineConfig, LmEngine, Seq

SLOTS = 4            # most live requests of a trace
PAGE = 64


def replay_engine(path: str, dtype: torch.dtype, max_tokens: int, device: str = "cuda:0", slots: int = SLOTS) -> LmEngine:
    """The engine of a model directory with a KV pool of ``max_tokens`` tokens (whole pages) and ``slots`` state slots;
    its scheduler thread is not started: the trace plans the steps."""
    from ..loaders.model import load_model
    from ..models.decoder import Decoder
    cfg, w, tok, _ = load_model(path, device, dtype)
    tokens = -(-max(max_tokens, 1) // PAGE) * PAGE
    ec = EngineConfig(ctx_size=tokens, max_seqs=slots, block_size=PAGE, kv_cache_tokens=tokens, prefix_cache=False,
                      max_batch_tokens=tokens, prefill_chunk=tokens, device=device)
    return LmEngine(Decoder(cfg, w, None, max_position=tokens + 8), tok, ec, start=False)


class TraceReplay:
    def __init__(self, engine: LmEngine):
        self.engine = engine
        self.live: Dict[str, Seq] = {}

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """One trace step; returns float32 logits [wanted, vocab] on the host, None when nothing is wanted."""
        items = []
        for e in entries:
            s = self.live.get(e["id"])
            if s is None:
                s = self.live[e["id"]] = self.engine.open_sequence(e["id"])
            items.append((s, [int(t) for t in e["tokens"]], [int(p) for p in e.get("want", [])]))
        items = [it for it in items if it[1]]
        out = self.engine.feed(items) if items else None
        if out is not None:
            out = out.float().cpu()
        if self.engine.device.type == "cuda":
            from ..ops import sm100
            code = sm100.Workspace.get(self.engine.device).check()
            if code:
                raise RuntimeError(f"a kernel of this step reported status {code}")
        for name in end:
            s = self.live.pop(name, None)
            if s is not None:
                self.engine.close_sequence(s)
        return out
