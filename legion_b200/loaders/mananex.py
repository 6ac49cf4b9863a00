"""Mananex checkpoints: ``config.json`` with ``architecture: "Mananex"`` and one entry per layer (sizes and constants of the
two mixers side by side, feed-forward kind and sizes or null), ``model.safetensors`` with tensors named ``l<i>.mix.left.*`` /
``l<i>.mix.right.*`` / ``l<i>.mlp.*`` / ``l<i>.rg<q>`` / ``l<i>.dwa``.

Everything that reads a layer's norm, except its feed-forward part, is stacked into one projection
(``ModelConfig.mix_columns``: q | k | v | head gates | recurrent q | forget gate | recurrent v | residual gates), and the
output projections of the two mixers into one matrix over their concatenated columns.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config import AttnSpec, DenseSpec, Hgrn2Spec, LayerSpec, ModelConfig, MoeSpec, ParallelSpec, RotarySpec
from ..models.weights import is_fp32_weight


def is_mananex(c: dict) -> bool:
    return c.get("architecture") == "Mananex"


def _mixer(kind: str, m: dict):
    if kind != "parallel":
        raise ValueError(f"Mananex: unknown mixer type {kind!r}")
    a, r = m["left"], m["right"]
    rot, mask = a.get("rot") or {}, a.get("mask") or {}
    return ParallelSpec(
        AttnSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                 window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0), qk_norm=False,
                 rot=RotarySpec(int(rot["dims"]), float(rot["base"])) if rot.get("dims") else None, sink=True, gate="head"),
        Hgrn2Spec(int(r["heads"]), int(r["dim"]), int(r["vdim"])), float(m["left_scale"]), float(m["right_scale"]))


def _mlp(f):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseSpec(int(f["ff"]), "silu", bias=True)
    if f["kind"] == "moe":
        return MoeSpec(int(f["router"]["experts"]), int(f["router"]["top"]), int(f["expert"]["ff"]), "silu",
                       router="biased_softmax")
    raise ValueError(f"Mananex: unknown feed-forward kind {f['kind']!r}")


def config_from_json(c: dict) -> ModelConfig:
    return ModelConfig(arch="mananex", hidden=int(c["width"]), vocab=int(c["vocab"]), rms_eps=float(c["norm"]["eps"]),
                       norm_offset=1.0, tie_embeddings=True, parallel_sublayers=True, residual_gate=True, depth_average=True,
                       layers=[LayerSpec(_mixer(x["type"], x["mixer"]), _mlp(x.get("mlp"))) for x in c["layers"]])


def load(ck, device, dtype) -> "tuple[ModelConfig, Dict[str, torch.Tensor]]":
    """``ck``: ``safetensors_io.Checkpoint``. Returns (config, canonical weights on ``device``)."""
    cfg = config_from_json(ck.config)
    get = lambda name: ck.get(name).to(device)                                  # noqa: E731
    cat = lambda *names: torch.cat([get(n) for n in names], 0)                  # noqa: E731
    w: Dict[str, torch.Tensor] = {"tok_embd": get("embed"), "output_norm": get("final.norm")}
    for il, spec in enumerate(cfg.layers):
        p, f = f"l{il}", spec.mlp
        a, r = f"{p}.mix.left", f"{p}.mix.right"
        w[f"{p}.attn_norm"] = get(f"{p}.norm1")
        col = cfg.mix_columns(il)
        rows = torch.zeros(col["end"], cfg.hidden, dtype=ck.get(f"{a}.q").dtype, device=device)
        sources = {"q": f"{a}.q", "k": f"{a}.k", "v": f"{a}.v", "g": f"{a}.g", "rq": f"{r}.q", "rf": f"{r}.f", "rv": f"{r}.v",
                   "rg1": f"{p}.rg1", "rg2": f"{p}.rg2"}
        for part, name in sources.items():
            if part in col:
                t = get(name)
                rows[col[part]:col[part] + t.shape[0]] = t
        w[f"{p}.mix.in"] = rows
        w[f"{p}.mix.o"] = torch.cat([get(f"{a}.o"), get(f"{r}.o")], 1)
        w[f"{p}.attn.sink"] = get(f"{a}.sink")
        w[f"{p}.hg.f_b"], w[f"{p}.hg.lower"], w[f"{p}.hg.norm"] = get(f"{r}.f.b"), get(f"{r}.lower"), get(f"{r}.norm")
        w[f"{p}.rg_b"] = get(f"{p}.rg1.b") if f is None else cat(f"{p}.rg1.b", f"{p}.rg2.b")
        w[f"{p}.dwa"] = get(f"{p}.dwa")
        if f is None:
            continue
        if f.kind == "dense":
            w[f"{p}.mlp.gate_up"], w[f"{p}.mlp.down"] = cat(f"{p}.mlp.gate", f"{p}.mlp.up"), get(f"{p}.mlp.down")
            w[f"{p}.mlp.gate_up_b"], w[f"{p}.mlp.down_b"] = cat(f"{p}.mlp.gate.b", f"{p}.mlp.up.b"), get(f"{p}.mlp.down.b")
            continue
        w[f"{p}.moe.router"], w[f"{p}.moe.router_bias"] = get(f"{p}.mlp.router"), get(f"{p}.mlp.router.b")
        w[f"{p}.moe.gate_up"] = torch.stack([cat(f"{p}.mlp.e{e}.gate", f"{p}.mlp.e{e}.up") for e in range(f.experts)])
        w[f"{p}.moe.down"] = torch.stack([get(f"{p}.mlp.e{e}.down") for e in range(f.experts)])
    out = {k: v.to(dtype=torch.float32 if is_fp32_weight(k) else dtype).contiguous() for k, v in w.items()}
    return cfg, out
