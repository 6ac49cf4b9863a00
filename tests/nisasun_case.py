"""Small Nisasun configurations, random weights for them, checkpoints on disk, and feeding schedules for engines."""
import json
import math
import os

import torch

from legion_b200.loaders.safetensors_io import save_file


def attention(heads, kv, dim, vdim, window, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window},
            "scale": scale if scale is not None else dim ** -0.5}


def state_space(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(left, right, mlp, ls=0.7, rs=0.6):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs}, "mlp": mlp}


def lightning(heads, dim, vdim, mlp, decay=None):
    return {"type": "lightning", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                      "decay": decay or [1 - 0.5 ** (1 + 1.3 * h) for h in range(heads)]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, count=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count,
                                                                                                      "keep": keep}}}


def config(width, vocab, streams, layers, eps=1e-5):
    return {"architecture": "Nisasun", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps},
            "layers": layers}


CASES = {
    # sizes that differ from each other and from layer to layer; a layer without feed-forward part
    "mixed": config(144, 160, 3, [
        parallel(attention(6, 3, 40, 24, 37), state_space(6, 24, 16, 2, 3, 3), moe(10, 3, 56, 5, 3)),
        lightning(3, 48, 64, None),
        parallel(attention(4, 1, 64, 80, 70), state_space(2, 48, 40, 1, 5, 2), dense(88), 1.2, 0.3),
        lightning(5, 32, 24, moe(6, 2, 40, 2, 1))]),
    # one stream, one group, one expert, one tap, a window of one token, sizes that no vector width divides
    "ones": config(90, 101, 1, [
        lightning(2, 13, 19, moe(3, 1, 27), [0.0, 1.0]),
        parallel(attention(2, 2, 21, 11, 1), state_space(1, 15, 9, 1, 1, 1), dense(33)),
        parallel(attention(3, 1, 17, 35, 5, 0.4), state_space(4, 7, 6, 4, 2, 2), None)]),
    # head sizes of real models: tensor-core tiles of 128, several value tiles
    "wide": config(256, 192, 4, [
        lightning(2, 128, 160, dense(256)),
        parallel(attention(4, 2, 200, 256, 130), state_space(4, 64, 128, 2, 4, 2), moe(8, 2, 64, 4, 2)),
        parallel(attention(8, 2, 128, 64, 200), state_space(2, 128, 128), dense(128))]),
}


def make_weights(cfg, seed=0, dtype=torch.bfloat16, decisive=False):
    """Random weights by checkpoint name. Head norms are scaled up so that single keys stand out among the scores.
    ``decisive``: corrections so far apart that rounding cannot change a routing choice (bf16 comparisons of whole
    models, where one flipped choice would change every later token)."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)                     # noqa: E731
    u = lambda *s: torch.rand(*s, generator=g)                      # noqa: E731
    W, S = cfg["width"], cfg["streams"]
    lin = lambda o, i, k=1.0: r(o, i) * k / math.sqrt(i)            # noqa: E731
    w = {"embed": r(cfg["vocab"], W), "final.norm": r(W) * 0.1, "head": lin(cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        w[p + ".norm1"] = r(W) * 0.1
        if layer["type"] == "lightning":
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            for n, o in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
                w[f"{p}.mix.{n}"] = lin(o, W)
            w[p + ".mix.norm"] = 1 + r(H * dv) * 0.1
            w[p + ".mix.o"] = lin(W, H * dv)
        else:
            a, s = m["left"], m["right"]
            b = p + ".mix.left"
            w[b + ".q"] = lin(a["heads"] * a["dim"], W)
            w[b + ".k"] = lin(a["kv_heads"] * a["dim"], W)
            w[b + ".v"] = lin(a["kv_heads"] * a["vdim"], W)
            w[b + ".q.norm"] = 2 + r(a["dim"]) * 0.2
            w[b + ".k.norm"] = 2 + r(a["dim"]) * 0.2
            w[b + ".o"] = lin(W, a["heads"] * a["vdim"])
            b = p + ".mix.right"
            inner, gn, H = s["heads"] * s["vdim"], s["groups"] * s["state"], s["heads"]
            w[b + ".in"] = lin(2 * inner + 2 * gn + H, W)
            w[b + ".conv"] = r(inner + 2 * gn, s["conv"]) * 0.5
            w[b + ".conv.b"] = r(inner + 2 * gn) * 0.2
            w[b + ".dt_bias"] = r(H) - 1
            w[b + ".A_log"] = torch.log(0.3 + 3 * u(H))
            w[b + ".D"] = 1 + r(H) * 0.2
            w[b + ".norm"] = 1 + r(inner) * 0.1
            w[b + ".o"] = lin(W, inner)
        f = layer["mlp"]
        for q in (1, 2)[:1 if f is None else 2]:
            w[f"{p}.hc{q}.in"] = (1 + r(S) * 0.3) / S
            w[f"{p}.hc{q}.out"] = 1 + r(S) * 0.3
            w[f"{p}.hc{q}.mix"] = torch.eye(S) * 0.8 + r(S, S) * 0.15
        if f is None:
            continue
        w[p + ".norm2"] = r(W) * 0.1
        parts = [p + ".mlp"]
        ff = f.get("ff")
        if f["kind"] == "moe":
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            parts = [f"{p}.mlp.e{e}" for e in range(E)]
            w[p + ".mlp.router"] = lin(E, W, 3.0)
            w[p + ".mlp.correction"] = r(E) * 0.3 - 0.3          # selection scores of either sign
            if decisive:
                w[p + ".mlp.correction"] = 2.0 * torch.randperm(E, generator=g) - E
        for b in parts:
            w[b + ".gate"], w[b + ".up"], w[b + ".down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    return {k: v.to(dtype).contiguous() for k, v in w.items()}


def write_checkpoint(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(weights, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def run_schedule(replay, seqs, schedule):
    """``schedule``: steps of [(name, tokens of this step)]. Feeds them, ends each sequence with its last token, and
    returns name -> logits [tokens, vocab] of everything."""
    at, got = {}, {}
    for n, step in enumerate(schedule):
        entries, end = [], []
        for name, c in step:
            lo = at.get(name, 0)
            entries.append({"id": name, "tokens": seqs[name][lo:lo + c], "want": list(range(c))})
            at[name] = lo + c
            if at[name] == len(seqs[name]):
                end.append(name)
        out, r = replay.step(entries, end), 0
        for name, c in step:
            got.setdefault(name, []).append(out[r:r + c])
            r += c
    return {k: torch.cat(v) for k, v in got.items()}


def errors(got, want):
    """Per position: RMS difference of the logits (mean taken off) over the RMS of the expected ones."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()
