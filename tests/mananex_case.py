"""Small Mananex configurations and random weights for them."""
import math

import torch


def left(heads, kv, dim, vdim, window, keep, dims, base=1e4, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5,
            "mask": {"size": window, "keep_first": keep}, "rot": {"dims": dims, "base": base}}


def right(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def layer(a, r, mlp, ls=0.7, rs=0.8):
    return {"type": "parallel", "mixer": {"left": a, "right": r, "left_scale": ls, "right_scale": rs}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Mananex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


CASES = {
    # sizes that differ from each other and from layer to layer, windows off every page and tile size, a layer without
    # feed-forward part, experts before dense parts
    "mixed": config(144, 160, [
        layer(left(6, 2, 40, 24, 37, 3, 24), right(3, 40, 56), moe(10, 3, 56)),
        layer(left(4, 4, 32, 48, 70, 6, 32, 3e3), right(5, 24, 32), dense(88), 1.2, 0.4),
        layer(left(2, 1, 64, 72, 129, 1, 10), right(2, 72, 96), None, 0.5, 1.1),
        layer(left(4, 2, 48, 40, 16, 2, 48), right(1, 128, 40), moe(6, 2, 40), 0.9, 0.9)]),
    # one head, one expert, a window of one token, no kept token, sizes that no vector width divides
    "ones": config(90, 101, [
        layer(left(1, 1, 21, 11, 9, 1, 10, scale=0.5), right(1, 13, 19), dense(33), 1.0, 1.0),
        layer(left(3, 1, 17, 35, 1, 2, 2, scale=0.4), right(2, 7, 5), moe(3, 1, 27), 0.3, 1.7),
        layer(left(2, 2, 13, 7, 25, 0, 12), right(1, 130, 3), moe(1, 1, 9), 1.1, 0.2)]),
    # head sizes of real models, windows and kept tokens beyond a tile, every expert chosen, wide heads
    "wide": config(256, 192, [
        layer(left(8, 2, 128, 64, 150, 140, 64), right(2, 128, 128), moe(8, 2, 64)),
        layer(left(4, 1, 96, 128, 300, 4, 96, 1e6), right(4, 64, 64), dense(320), 0.5, 0.5),
        layer(left(2, 2, 200, 256, 64, 64, 128), right(1, 192, 136), moe(8, 8, 40), 0.6, 1.0),
        layer(left(16, 2, 64, 64, 500, 7, 64), right(3, 64, 128), moe(16, 4, 64), 0.8, 0.6)]),
}


def make_weights(cfg, seed=0, dtype=torch.bfloat16, decisive=False):
    """Random weights by checkpoint name. Queries and keys are scaled up so that single keys stand out among the scores, sinks
    take a visible share; forget gates spread from short to long memories, depth averages mix results of either sign.
    ``decisive``: router rows so large that rounding hardly changes a choice."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)                     # noqa: E731
    u = lambda *s: torch.rand(*s, generator=g)                      # noqa: E731
    W = cfg["width"]
    lin = lambda o, i, k=1.0: r(o, i) * k / math.sqrt(i)            # noqa: E731
    w = {"embed": r(cfg["vocab"], W), "final.norm": r(W) * 0.1}
    for i, spec in enumerate(cfg["layers"]):
        p, f = f"l{i}", spec["mlp"]
        a, s = spec["mixer"]["left"], spec["mixer"]["right"]
        w[p + ".norm1"] = r(W) * 0.1
        b = p + ".mix.left"
        w[b + ".q"], w[b + ".k"] = lin(a["heads"] * a["dim"], W, 1.6), lin(a["kv_heads"] * a["dim"], W, 1.6)
        w[b + ".v"], w[b + ".g"] = lin(a["kv_heads"] * a["vdim"], W), lin(a["heads"], W)
        w[b + ".sink"], w[b + ".o"] = 1 + r(a["heads"]), lin(W, a["heads"] * a["vdim"])
        b = p + ".mix.right"
        nk = s["heads"] * s["dim"]
        w[b + ".q"], w[b + ".f"], w[b + ".v"] = lin(nk, W), lin(nk, W), lin(s["heads"] * s["vdim"], W)
        w[b + ".f.b"] = 6 * u(nk) - 1
        w[b + ".lower"] = (u(nk) - 0.2).clamp(min=0)                # some bounds are zero
        w[b + ".norm"], w[b + ".o"] = 1 + r(s["vdim"]) * 0.2, lin(W, s["heads"] * s["vdim"])
        w[p + ".rg1"], w[p + ".rg1.b"] = lin(W, W), 0.5 + r(W) * 0.5
        w[p + ".dwa"] = torch.cat([r(i + 1) * 0.25, 1 + r(1) * 0.2])
        if f is None:
            continue
        w[p + ".rg2"], w[p + ".rg2.b"] = lin(W, W), 0.5 + r(W) * 0.5
        if f["kind"] == "dense":
            for n, o, k in (("gate", f["ff"], W), ("up", f["ff"], W), ("down", W, f["ff"])):
                w[f"{p}.mlp.{n}"], w[f"{p}.mlp.{n}.b"] = lin(o, k), r(o) * 0.3
            continue
        E = f["router"]["experts"]
        w[p + ".mlp.router"], w[p + ".mlp.router.b"] = lin(E, W, 8.0 if decisive else 1.5), r(E)
        for e in range(E):
            n, ff = f"{p}.mlp.e{e}", f["expert"]["ff"]
            w[n + ".gate"], w[n + ".up"], w[n + ".down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    return {k: v.to(dtype).contiguous() for k, v in w.items()}
