"""Small Pemezen configurations and random weights for them."""
import math

import torch


def latent(heads, dim, rot_dim, vdim, rank, mlp, per_head=False, base=1e4, factor=4.0, original=64, fast=32.0, slow=1.0,
           scale=None):
    return {"type": "latent_attention_2" if per_head else "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
                      "rot": {"base": base, "dims": rot_dim, "scaling": {"factor": factor, "original": original, "fast": fast,
                                                                        "slow": slow}}}}


def rglru(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, groups, taps, layers, emb=2.0, cap=9.0, eps=1e-5):
    return {"architecture": "Pemezen", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups},
            "canon": {"taps": taps}, "embedding": {"scale": emb}, "logit_softcap": cap, "layers": layers}


CASES = {
    # sizes that differ from each other and from layer to layer; a layer without feed-forward part
    "mixed": config(144, 160, 3, 3, [
        latent(6, 40, 24, 32, 72, dense(200), per_head=True),
        rglru(96, 3, 5, dense(88)),
        latent(2, 64, 16, 48, 96, None, base=3e3, factor=2.0, original=300),
        rglru(64, 1, 2, dense(136))]),
    # one group, one tap, one head, one block, sizes that no vector width divides, no scaling of anything
    "ones": config(90, 101, 1, 1, [
        rglru(21, 1, 1, dense(33)),
        latent(1, 13, 6, 11, 19, dense(27), factor=1.0),
        latent(3, 1, 2, 1, 7, dense(50), per_head=True, original=20000, scale=0.4),
        rglru(35, 35, 3, None)], emb=1.0, cap=30.0),
    # head and latent sizes of real models; more heads than a query tile holds, head counts that do not divide it
    "wide": config(256, 192, 8, 4, [
        latent(16, 128, 64, 128, 512, dense(320), original=128),
        rglru(320, 2, 4, dense(256)),
        latent(5, 64, 32, 72, 256, dense(128), per_head=True),
        latent(70, 16, 8, 8, 136, dense(64))]),
}


def make_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights by checkpoint name. Query and latent projections are scaled up so that single keys stand out among
    the scores, decays spread from fast to slow."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)                     # noqa: E731
    u = lambda *s: torch.rand(*s, generator=g)                      # noqa: E731
    W, K = cfg["width"], cfg["canon"]["taps"]
    lin = lambda o, i, k=1.0: r(o, i) * k / math.sqrt(i)            # noqa: E731
    norm = lambda n: 1 + r(n) * 0.2                                 # noqa: E731
    w = {"embed": r(cfg["vocab"], W), "final.norm": norm(W), "head": lin(cfg["vocab"], W, 4.0)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer["mlp"]
        for q in (1, 2)[:1 if f is None else 2]:
            w[f"{p}.norm{q}"], w[f"{p}.norm{q}b"] = norm(W), norm(W)
            w[f"{p}.canon{q}"] = r(W, K) * 0.4
        b = p + ".mix"
        if layer["type"] == "rglru":
            n, d = m["width"], m["width"] // m["blocks"]
            w[b + ".y"], w[b + ".y.b"], w[b + ".x"], w[b + ".x.b"] = lin(n, W), r(n) * 0.3, lin(n, W), r(n) * 0.3
            w[b + ".conv"], w[b + ".conv.b"] = r(n, m["conv"]) * 0.5, r(n) * 0.2
            for x in ("ra", "ri"):
                w[f"{b}.{x}"], w[f"{b}.{x}.b"] = r(m["blocks"], d, d) * 1.5 / math.sqrt(d), r(m["blocks"], d) * 0.5
            w[b + ".lam"] = torch.log(torch.expm1(0.002 + 0.3 * u(n) ** 3))
            w[b + ".o"] = lin(W, n)
        else:
            H, L, hd = m["heads"], m["kv_rank"], m["dim"] + m["rot_dim"]
            w[b + ".q"], w[b + ".dkv"], w[b + ".dkv.norm"] = lin(H * hd, W, 1.6), lin(L + m["rot_dim"], W, 1.3), norm(L)
            w[b + ".uk"], w[b + ".uv"] = lin(H * m["dim"], L, 1.6), lin(H * m["vdim"], L)
            w[b + ".g"] = lin(H if layer["type"].endswith("_2") else H * m["vdim"], W)
            w[b + ".o"] = lin(W, H * m["vdim"])
        if f is not None:
            w[p + ".mlp.up"], w[p + ".mlp.down"], w[p + ".mlp.act"] = lin(f["ff"], W), lin(W, f["ff"]), r(2) * 0.7
    return {k: v.to(dtype).contiguous() for k, v in w.items()}
