"""Gurozen checkpoints: ``config.json`` with ``architecture: "Gurozen"`` and one entry per layer (mixer type and sizes,
feed-forward kind and sizes or null), ``model.safetensors`` with tensors named ``l<i>.mix.*`` / ``l<i>.mlp.*``.

Every size and constant of a layer is its own, so the configuration is a list of ``LayerSpec``, one per layer run (the
passes of ``loop`` share weights). The width of the low-rank projections stands in the tensors' shapes only. On the way in
the projections that read one input are stacked, ``A_log`` becomes ``-exp(A_log)``, the shared expert's gate becomes the
last row of the router, and the shared expert itself is cut into experts of the routed width.
"""
from __future__ import annotations

from typing import Dict

import torch
import torch.nn.functional as F

from ..config import AttnSpec, ChannelDeltaSpec, DenseSpec, LayerSpec, LoopSpec, ModelConfig, MoeSpec, RotarySpec
from ..models.weights import is_fp32_weight


def is_gurozen(c: dict) -> bool:
    return c.get("architecture") == "Gurozen"


def _rotary(r):
    if not r or not int(r["dims"]):
        return None
    s = r.get("scaling")
    if not s:
        return RotarySpec(int(r["dims"]), float(r["base"]), layout="half")
    return RotarySpec(int(r["dims"]), float(r["base"]), float(s["factor"]), float(s["original"]), scaling="llama3",
                      low=float(s["low"]), high=float(s["high"]), layout="half")


def _mixer(kind: str, m: dict):
    if kind == "attention":
        return AttnSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                        norm_over="all", bias=True, conv=int(m["conv"]), rot=_rotary(m.get("rot")),
                        softcap=float(m.get("softcap") or 0.0))
    if kind == "channel_delta":
        return ChannelDeltaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
    raise ValueError(f"Gurozen: unknown mixer type {kind!r}")


def _mlp(f):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseSpec(int(f["ff"]), "silu")
    if f["kind"] == "moe":
        r, g, shared = f["router"], f["router"].get("groups") or {"count": 1, "keep": 1}, f.get("shared")
        return MoeSpec(int(r["experts"]), int(r["top"]), int(f["expert"]["ff"]), "relu2", router="sigmoid", renorm="sum",
                       scale=float(r["scale"]), n_group=int(g["count"]), keep_group=int(g["keep"]), group_top=2,
                       shared_ff=int(shared["ff"]) if shared else 0, shared_gate=bool(shared))
    raise ValueError(f"Gurozen: unknown feed-forward kind {f['kind']!r}")


def config_from_json(c: dict) -> ModelConfig:
    layers = [LayerSpec(_mixer(x["type"], x["mixer"]), _mlp(x.get("mlp"))) for x in c["layers"]]
    loop = c.get("loop")
    if loop:
        loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        layers = loop.expand(layers)
    return ModelConfig(arch="gurozen", hidden=int(c["width"]), vocab=int(c["vocab"]), rms_eps=float(c["norm"]["eps"]),
                       norm_offset=1.0, tie_embeddings=True, embed_norm=True, residual_mult=float(c["residual_mult"]),
                       logit_scale=float(c["logit_scale"]), layers=layers, loop=loop or None)


def load(ck, device, dtype) -> "tuple[ModelConfig, Dict[str, torch.Tensor]]":
    """``ck``: ``safetensors_io.Checkpoint``. Returns (config, canonical weights on ``device``)."""
    cfg = config_from_json(ck.config)
    get = lambda name: ck.get(name).to(device)                                  # noqa: E731
    cat = lambda *names: torch.cat([get(n) for n in names], 0)                  # noqa: E731
    w: Dict[str, torch.Tensor] = {"tok_embd": get("embed"), "output_norm": get("final.norm"), "embed_norm": get("embed.norm")}
    if cfg.loop is not None:
        w["loop_in"] = get("loop.in")
    for il, spec in enumerate(cfg.layers):
        p, m, f = f"l{cfg.weight_layer(il)}", spec.mixer, spec.mlp
        b = f"{p}.mix"
        if m.kind == "channel_delta":
            m.rank = -(-max(ck.get(f"{b}.a1").shape[0], ck.get(f"{b}.g1").shape[0]) // 8) * 8
        if f"{p}.attn_norm" in w:
            continue                                                            # a further pass of the same layer
        w[f"{p}.attn_norm"] = get(f"{p}.norm1")
        if m.kind == "attn":
            w[f"{p}.mix.in"], w[f"{p}.attn.in_b"] = cat(f"{b}.q", f"{b}.k", f"{b}.v"), cat(f"{b}.q.b", f"{b}.k.b", f"{b}.v.b")
            w[f"{p}.attn.q_norm"], w[f"{p}.attn.k_norm"] = get(f"{b}.q.norm"), get(f"{b}.k.norm")
            if m.conv:
                w[f"{p}.attn.conv_w"] = cat(f"{b}.q.conv", f"{b}.k.conv", f"{b}.v.conv").t()
            w[f"{p}.attn.o"] = get(f"{b}.o")
        else:
            col = m.in_columns()
            rows = torch.zeros(col["end"], cfg.hidden, dtype=ck.get(f"{b}.q").dtype, device=device)
            for part in ("q", "k", "v", "b", "a1", "g1"):
                t = get(f"{b}.{part}")
                rows[col[part]:col[part] + t.shape[0]] = t
            w[f"{p}.cd.in"] = rows
            w[f"{p}.cd.conv_w"] = cat(f"{b}.q.conv", f"{b}.k.conv", f"{b}.v.conv").t()
            w[f"{p}.cd.low"] = torch.cat([F.pad(t, (0, m.rank - t.shape[1])) for t in (get(f"{b}.a2"), get(f"{b}.g2"))], 0)
            w[f"{p}.cd.A"] = -torch.exp(get(f"{b}.A_log").double())
            w[f"{p}.cd.dt_bias"], w[f"{p}.cd.norm"], w[f"{p}.cd.out"] = get(f"{b}.dt_bias"), get(f"{b}.norm"), get(f"{b}.o")
        if f is None:
            continue
        w[f"{p}.ffn_norm"] = get(f"{p}.norm2")
        if f.kind == "dense":
            w[f"{p}.mlp.gate_up"], w[f"{p}.mlp.down"] = cat(f"{p}.mlp.gate", f"{p}.mlp.up"), get(f"{p}.mlp.down")
            continue
        up = [get(f"{p}.mlp.e{e}.up") for e in range(f.experts)]
        down = [get(f"{p}.mlp.e{e}.down") for e in range(f.experts)]
        w[f"{p}.moe.router"] = get(f"{p}.mlp.router")
        if f.shared_ff:
            s, pad = f"{p}.mlp.shared", f.shared_slots() * f.ff - f.shared_ff
            w[f"{p}.moe.router"] = cat(f"{p}.mlp.router", f"{s}.sg")
            up += F.pad(get(f"{s}.up"), (0, 0, 0, pad)).split(f.ff, 0)
            down += F.pad(get(f"{s}.down"), (0, pad)).split(f.ff, 1)
        w[f"{p}.moe.gate_up"], w[f"{p}.moe.down"] = torch.stack(up), torch.stack(down)
    out = {k: v.to(dtype=torch.float32 if is_fp32_weight(k) else dtype).contiguous() for k, v in w.items()}
    return cfg, out
