"""Nisasun checkpoints: ``config.json`` with ``architecture: "Nisasun"`` and one entry per layer (mixer type and sizes,
feed-forward kind and sizes), ``model.safetensors`` with tensors named ``l<i>.mix.*`` / ``l<i>.mlp.*`` / ``l<i>.hc<q>.*``.

Every size and constant of a layer is its own, so the configuration is a list of ``LayerSpec``; the projections that
read the same input are stacked on the way in, and ``A_log`` becomes ``-exp(A_log)``.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config import AttnSpec, DenseSpec, LayerSpec, LightningSpec, ModelConfig, MoeSpec, ParallelSpec, SsdSpec
from ..models.weights import is_fp32_weight


def is_nisasun(c: dict) -> bool:
    return c.get("architecture") == "Nisasun"


def _mixer(kind: str, m: dict):
    if kind == "lightning":
        return LightningSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), [float(d) for d in m["decay"]])
    if kind == "parallel":
        a, r = m["left"], m["right"]
        return ParallelSpec(
            AttnSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]),
                     window=int(a["mask"]["size"])),
            SsdSpec(int(r["heads"]), int(r["vdim"]), int(r["state"]), int(r["groups"]), int(r["conv"]),
                    int(r["norm_groups"])),
            float(m["left_scale"]), float(m["right_scale"]))
    raise ValueError(f"Nisasun: unknown mixer type {kind!r}")


def _mlp(f):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseSpec(int(f["ff"]), "gelu_tanh")
    if f["kind"] == "moe":
        r = f["router"]
        return MoeSpec(int(r["experts"]), int(r["top"]), int(f["expert"]["ff"]), "silu", router="softmax_bias",
                       correction=True, renorm=False, n_group=int(r["groups"]["count"]),
                       keep_group=int(r["groups"]["keep"]), group_top=1)
    raise ValueError(f"Nisasun: unknown feed-forward kind {f['kind']!r}")


def config_from_json(c: dict) -> ModelConfig:
    return ModelConfig(arch="nisasun", hidden=int(c["width"]), vocab=int(c["vocab"]), rms_eps=float(c["norm"]["eps"]),
                       norm_offset=1.0, hyper_streams=int(c["streams"]), hyper_mode="static",
                       layers=[LayerSpec(_mixer(x["type"], x["mixer"]), _mlp(x["mlp"])) for x in c["layers"]])


def load(ck, device, dtype) -> "tuple[ModelConfig, Dict[str, torch.Tensor]]":
    """``ck``: ``safetensors_io.Checkpoint``. Returns (config, canonical weights on ``device``)."""
    cfg = config_from_json(ck.config)
    get = lambda name: ck.get(name).to(device)                                  # noqa: E731
    cat = lambda *names: torch.cat([get(n) for n in names], 0)                  # noqa: E731
    w: Dict[str, torch.Tensor] = {"tok_embd": get("embed"), "output_norm": get("final.norm"), "output": get("head")}
    for il, spec in enumerate(cfg.layers):
        p = f"l{il}"
        w[f"{p}.attn_norm"] = get(f"{p}.norm1")
        for q, which in ((1, "hca"), (2, "hcf"))[:1 if spec.mlp is None else 2]:
            for leaf in ("in", "out", "mix"):
                w[f"{p}.{which}.st_{leaf}"] = get(f"{p}.hc{q}.{leaf}")
        m = f"{p}.mix"
        if spec.mixer.kind == "lightning":
            w[f"{p}.lin.qkvg"] = cat(*(f"{m}.{x}" for x in "qkvg"))
            w[f"{p}.lin.norm"] = get(f"{m}.norm")
            w[f"{p}.lin.out"] = get(f"{m}.o")
        else:
            a, r = f"{m}.left", f"{m}.right"
            w[f"{p}.mix.in"] = cat(f"{a}.q", f"{a}.k", f"{a}.v", f"{r}.in")
            w[f"{p}.attn.q_norm"], w[f"{p}.attn.k_norm"] = get(f"{a}.q.norm"), get(f"{a}.k.norm")
            w[f"{p}.attn.o"] = get(f"{a}.o")
            w[f"{p}.ssm.conv_w"], w[f"{p}.ssm.conv_b"] = get(f"{r}.conv"), get(f"{r}.conv.b")
            w[f"{p}.ssm.A"] = -torch.exp(get(f"{r}.A_log").float())
            w[f"{p}.ssm.D"], w[f"{p}.ssm.dt_bias"] = get(f"{r}.D"), get(f"{r}.dt_bias")
            w[f"{p}.ssm.norm"], w[f"{p}.ssm.out"] = get(f"{r}.norm"), get(f"{r}.o")
        f = spec.mlp
        if f is None:
            continue
        w[f"{p}.ffn_norm"] = get(f"{p}.norm2")
        if f.kind == "dense":
            w[f"{p}.mlp.gate_up"] = cat(f"{p}.mlp.gate", f"{p}.mlp.up")
            w[f"{p}.mlp.down"] = get(f"{p}.mlp.down")
        else:
            w[f"{p}.moe.router"] = get(f"{p}.mlp.router")
            w[f"{p}.moe.router_bias"] = get(f"{p}.mlp.correction")
            w[f"{p}.moe.gate_up"] = torch.stack([cat(f"{p}.mlp.e{e}.gate", f"{p}.mlp.e{e}.up") for e in range(f.experts)])
            w[f"{p}.moe.down"] = torch.stack([get(f"{p}.mlp.e{e}.down") for e in range(f.experts)])
    out = {k: v.to(dtype=torch.float32 if is_fp32_weight(k) else dtype).contiguous() for k, v in w.items()}
    return cfg, out
