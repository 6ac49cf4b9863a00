"""Pemezen checkpoints: ``config.json`` with ``architecture: "Pemezen"`` and one entry per layer (mixer type and sizes,
feed-forward size or null), ``model.safetensors`` with tensors named ``l<i>.mix.*`` / ``l<i>.mlp.*`` / ``l<i>.canon<q>``.

Every size and constant of a layer is its own, so the configuration is a list of ``LayerSpec``. On the way in the
projections that read one input are stacked, the key projection of the latent is transposed per head (queries are moved
into the latent space, so only latents are cached), and constants of the recurrence and the activation are evaluated:
``lam`` becomes -8 softplus(lam), the two numbers of xIELU become softplus(p) and 1/2 + softplus(q).
"""
from __future__ import annotations

from typing import Dict

import torch
import torch.nn.functional as F

from ..config import DenseSpec, LatentSpec, LayerSpec, ModelConfig, RgLruSpec, RotarySpec
from ..models.weights import is_fp32_weight, latent_in_rows

GATES = {"latent_attention": "channel", "latent_attention_2": "head"}
DECAY = -8.0            # log decay of an open recurrence gate, per softplus(lam)


def is_pemezen(c: dict) -> bool:
    return c.get("architecture") == "Pemezen"


def _mixer(kind: str, m: dict):
    if kind in GATES:
        r = m["rot"]
        s = r.get("scaling")
        rot = RotarySpec(int(r["dims"]), float(r["base"]))
        if s:
            rot = RotarySpec(int(r["dims"]), float(r["base"]), float(s["factor"]), float(s["original"]), float(s["fast"]),
                             float(s["slow"]))
        return LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                          float(m["scale"]), rot, GATES[kind])
    if kind == "rglru":
        return RgLruSpec(int(m["width"]), int(m["blocks"]), int(m["conv"]))
    raise ValueError(f"Pemezen: unknown mixer type {kind!r}")


def _mlp(f):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseSpec(int(f["ff"]), "xielu")
    raise ValueError(f"Pemezen: unknown feed-forward kind {f['kind']!r}")


def config_from_json(c: dict) -> ModelConfig:
    return ModelConfig(arch="pemezen", hidden=int(c["width"]), vocab=int(c["vocab"]), rms_eps=float(c["norm"]["eps"]),
                       sandwich_norm=True, norm_groups=int(c["norm"]["groups"]), input_conv=int(c["canon"]["taps"]),
                       embed_scale=float(c["embedding"]["scale"]), logit_softcap=float(c.get("logit_softcap") or 0.0),
                       layers=[LayerSpec(_mixer(x["type"], x["mixer"]), _mlp(x.get("mlp"))) for x in c["layers"]])


def load(ck, device, dtype) -> "tuple[ModelConfig, Dict[str, torch.Tensor]]":
    """``ck``: ``safetensors_io.Checkpoint``. Returns (config, canonical weights on ``device``)."""
    cfg = config_from_json(ck.config)
    get = lambda name: ck.get(name).to(device)                                  # noqa: E731
    cat = lambda *names: torch.cat([get(n) for n in names], 0)                  # noqa: E731
    w: Dict[str, torch.Tensor] = {"tok_embd": get("embed"), "output_norm": get("final.norm"), "output": get("head")}
    for il, spec in enumerate(cfg.layers):
        p, m, b = f"l{il}", spec.mixer, f"l{il}.mix"
        for q, which in ((1, "attn"), (2, "ffn"))[:1 if spec.mlp is None else 2]:
            w[f"{p}.{which}_norm"], w[f"{p}.{which}_post_norm"] = get(f"{p}.norm{q}"), get(f"{p}.norm{q}b")
            w[f"{p}.{which}_taps"] = get(f"{p}.canon{q}").t()
        if m.kind == "latent":
            parts = [f"{b}.q", f"{b}.dkv"] + ([f"{b}.g"] if m.gate != "none" else [])
            x = cat(*parts)
            w[f"{p}.lat.in"] = F.pad(x, (0, 0, 0, latent_in_rows(m) - x.shape[0]))
            w[f"{p}.lat.norm"] = get(f"{b}.dkv.norm")
            w[f"{p}.lat.uk"] = get(f"{b}.uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2).reshape(-1, m.dim)
            w[f"{p}.lat.uv"], w[f"{p}.lat.o"] = get(f"{b}.uv"), get(f"{b}.o")
        else:
            d = m.width // m.blocks
            w[f"{p}.lru.in"], w[f"{p}.lru.in_b"] = cat(f"{b}.y", f"{b}.x"), cat(f"{b}.y.b", f"{b}.x.b")
            w[f"{p}.lru.conv_w"], w[f"{p}.lru.conv_b"] = get(f"{b}.conv"), get(f"{b}.conv.b")
            w[f"{p}.lru.gates"] = torch.stack([get(f"{b}.ra"), get(f"{b}.ri")], 1).reshape(-1, d)
            w[f"{p}.lru.gates_b"] = torch.stack([get(f"{b}.ra.b"), get(f"{b}.ri.b")], 1).reshape(-1)
            w[f"{p}.lru.log_decay"] = DECAY * F.softplus(get(f"{b}.lam").double())
            w[f"{p}.lru.out"] = get(f"{b}.o")
        if spec.mlp is not None:
            w[f"{p}.mlp.up"], w[f"{p}.mlp.down"] = get(f"{p}.mlp.up"), get(f"{p}.mlp.down")
            w[f"{p}.mlp.act"] = F.softplus(get(f"{p}.mlp.act").double()) + torch.tensor([0.0, 0.5], dtype=torch.float64,
                                                                                       device=device)
    out = {k: v.to(dtype=torch.float32 if is_fp32_weight(k) else dtype).contiguous() for k, v in w.items()}
    return cfg, out
