"""Small Gurozen configurations and random weights for them."""
import math

import torch


def rot(dims, base=1e4, factor=4.0, low=1.0, high=4.0, original=96):
    return {"dims": dims, "base": base, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}


def attention(heads, kv, dim, vdim, mlp, conv=3, r=None, cap=20.0, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "rot": r or rot(dim),
                      "scale": scale if scale is not None else dim ** -0.5, "softcap": cap}}


def delta(heads, kv, dim, vdim, mlp, conv=4):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared, count=1, keep=1, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def config(width, vocab, layers, loop=None, mult=0.7, logit=1.5, eps=1e-5):
    c = {"architecture": "Gurozen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
         "logit_scale": logit, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # sizes that differ from each other and from layer to layer, fewer key heads than heads, a shared expert that is no
    # multiple of the routed width, a layer without feed-forward part; three passes of two layers
    "mixed": config(144, 160, [
        delta(6, 3, 40, 24, moe(10, 3, 56, 72, 5, 2)),
        attention(6, 2, 40, 56, dense(88), conv=4, r=rot(24)),
        delta(4, 1, 48, 72, None, conv=2),
        attention(4, 4, 64, 32, moe(6, 2, 40, 120, 3, 2), r=rot(64, 3e3, 8.0, 1.0, 2.0, 40))], loop=(1, 3, 3)),
    # one head, one expert, one tap, one pass from the first layer on, sizes that no vector width divides
    "ones": config(90, 101, [
        delta(1, 1, 13, 19, moe(3, 1, 27, 27), conv=1),
        attention(1, 1, 21, 11, moe(1, 1, 9, 5), conv=1, r=rot(10, factor=1.0), cap=5.0),
        delta(2, 2, 7, 5, dense(33), conv=6),
        attention(3, 1, 17, 35, None, conv=5, r=rot(2), scale=0.4)], loop=(0, 4, 1), mult=1.0, logit=1.0),
    # head sizes of real models, many taps of nothing else: tensor-core tiles, several experts' worth of shared expert
    "wide": config(256, 192, [
        attention(8, 2, 128, 64, moe(8, 2, 64, 256, 4, 2), r=rot(128, original=64)),
        delta(3, 3, 128, 128, dense(320)),
        attention(4, 1, 200, 256, moe(16, 4, 64, 64, 4, 1), conv=2, r=rot(96)),
        delta(2, 1, 192, 136, moe(8, 8, 40, 24), conv=3)], loop=(2, 4, 2), mult=0.4),
}


def make_weights(cfg, seed=0, dtype=torch.bfloat16, decisive=False):
    """Random weights by checkpoint name. Query and key norms are scaled up so that single keys stand out among the scores;
    decays spread from fast to slow, channel by channel. ``decisive``: router rows so large that rounding hardly changes a
    choice."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)                     # noqa: E731
    u = lambda *s: torch.rand(*s, generator=g)                      # noqa: E731
    W = cfg["width"]
    lin = lambda o, i, k=1.0: r(o, i) * k / math.sqrt(i)            # noqa: E731
    w = {"embed": r(cfg["vocab"], W), "embed.norm": r(W) * 0.2, "final.norm": r(W) * 0.1}
    if cfg.get("loop"):
        w["loop.in"] = lin(W, 2 * W)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer["mlp"]
        b = p + ".mix"
        w[p + ".norm1"] = r(W) * 0.1
        H, G, dk, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        if layer["type"] == "attention":
            for n, o in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                w[f"{b}.{n}"], w[f"{b}.{n}.b"], w[f"{b}.{n}.conv"] = lin(o, W), r(o) * 0.3, r(o, K) * 0.6
            w[b + ".q.norm"], w[b + ".k.norm"] = 2 + r(H * dk) * 0.2, 2 + r(G * dk) * 0.2
        else:
            for n, o in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                w[f"{b}.{n}"], w[f"{b}.{n}.conv"] = lin(o, W), r(o, K) * 0.8
            w[b + ".b"] = lin(H, W)
            w[b + ".a1"], w[b + ".a2"] = lin(min(dk, 11), W), lin(H * dk, min(dk, 11))
            w[b + ".g1"], w[b + ".g2"] = lin(min(dv, 5), W), lin(H * dv, min(dv, 5), 2.0)
            w[b + ".A_log"] = torch.log(0.02 + 2 * u(H) ** 2)
            w[b + ".dt_bias"] = 4 * u(H * dk) - 4
            w[b + ".norm"] = 1 + r(dv) * 0.2
        w[b + ".o"] = lin(W, H * dv)
        if f is None:
            continue
        w[p + ".norm2"] = r(W) * 0.1
        if f["kind"] == "dense":
            w[p + ".mlp.gate"], w[p + ".mlp.up"], w[p + ".mlp.down"] = lin(f["ff"], W), lin(f["ff"], W), lin(W, f["ff"])
            continue
        w[p + ".mlp.router"] = lin(f["router"]["experts"], W, 8.0 if decisive else 1.5)
        for n, ff in [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + [("shared", f["shared"]["ff"])]:
            w[f"{p}.mlp.{n}.up"], w[f"{p}.mlp.{n}.down"] = lin(ff, W), lin(W, ff)
        w[p + ".mlp.shared.sg"] = lin(1, W, 2.0)
    return {k: v.to(dtype).contiguous() for k, v in w.items()}
