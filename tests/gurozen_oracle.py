"""Plain, slow implementation of the Gurozen design, one function per mechanism, written from its equations.

It shares no code with the product path: float64 (or the dtype of the inputs) tensor arithmetic, one sequence at a time,
one token at a time wherever a recurrence or a convolution is involved. ``cfg`` is the raw ``config.json`` dictionary and
``w`` maps the checkpoint's tensor names to tensors.
"""
import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def model_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def short_conv(u, taps):
    """Causal depth-wise convolution; the last column of ``taps`` weighs the current token; u [T, channels]."""
    K = taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def frequencies(rot):
    """Rotation frequency per pair, with the stretched low frequencies of Llama 3.1."""
    out, s = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        if s:
            wave = 2 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                m = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - m) * f / s["factor"] + m * f
        out.append(f)
    return out


def rotate(x, positions, rot):
    """x [T, heads, >= dims]: column i turns with column i + dims / 2, by the position times the pair's frequency."""
    y = x.clone()
    half = rot["dims"] // 2
    for i, f in enumerate(frequencies(rot)):
        for t, p in enumerate(positions):
            c, s = math.cos(p * f), math.sin(p * f)
            u, v = x[t, :, i], x[t, :, i + half]
            y[t, :, i], y[t, :, i + half] = u * c - v * s, v * c + u * s
    return y


def softmax_heads(q, k, v, scale, cap=None):
    """q [Tq, H, d] of the last Tq of T positions, k [T, G, d], v [T, G, dv]: capped causal attention, [Tq, H, dv]."""
    Tq, H, T, G = q.shape[0], q.shape[1], k.shape[0], k.shape[1]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T - Tq, T)[:, None], -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append((e / e.sum(-1, keepdim=True)) @ v[:, h // (H // G)])
    return torch.stack(out, 1)


def qkv_rows(h, w, p, m, eps):
    """Projection, bias, short convolution, norm over the whole of q and of k, heads, rotation."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    u = {n: short_conv(h @ w[f"{p}.{n}"].T + w[f"{p}.{n}.b"], w[f"{p}.{n}.conv"]) for n in "qkv"}
    q = (rms(u["q"], eps) * w[p + ".q.norm"]).reshape(T, H, m["dim"])
    k = (rms(u["k"], eps) * w[p + ".k.norm"]).reshape(T, G, m["dim"])
    return rotate(q, range(T), m["rot"]), rotate(k, range(T), m["rot"]), u["v"].reshape(T, G, m["vdim"])


def attention(h, w, p, m, eps):
    q, k, v = qkv_rows(h, w, p, m, eps)
    return softmax_heads(q, k, v, m["scale"], m.get("softcap")).reshape(h.shape[0], -1) @ w[p + ".o"].T


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, S=None):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H]: the state's rows decay per key channel, then the value that k reads
    moves towards v by beta; the read-out sees the write. Returns (o [T, H, dv], last S [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S
    out = []
    for t in range(T):
        rows = []
        for h in range(H):
            M = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - M.T @ k[t, h])
            rows.append(M + torch.outer(k[t, h], u))
        S = torch.stack(rows)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def decay(a, A_log, dt_bias, heads):
    """a [T, heads * dim] before bias: exp(-exp(A_log) softplus(a + dt_bias)) as [T, heads, dim]."""
    z = softplus(a + dt_bias).reshape(a.shape[0], heads, -1)
    return torch.exp(-torch.exp(A_log)[None, :, None] * z)


def channel_delta(h, w, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (silu(short_conv(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"])) for n in "qkv")
    per_head = lambda x: unit(x.reshape(T, G, m["dim"])).repeat_interleave(H // G, 1)      # noqa: E731
    q, k = per_head(q) * m["dim"] ** -0.5, per_head(k)
    beta = sigmoid(h @ w[p + ".b"].T)
    g = decay((h @ w[p + ".a1"].T) @ w[p + ".a2"].T, w[p + ".A_log"], w[p + ".dt_bias"], H)
    o, _ = delta_rule(q, k, v.reshape(T, H, m["vdim"]), g, beta)
    gate = sigmoid((h @ w[p + ".g1"].T) @ w[p + ".g2"].T).reshape(o.shape)
    return (rms(o, eps) * w[p + ".norm"] * gate).reshape(T, -1) @ w[p + ".o"].T


def gated_ffn(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def square_relu_ffn(h, w, p):
    return torch.clamp(h @ w[p + ".up"].T, min=0) ** 2 @ w[p + ".down"].T


def route(z, router):
    """Logits z [experts] of one token -> {expert: weight}."""
    s = sigmoid(z)
    E, n = z.shape[0], router["groups"]["count"]
    size = E // n
    total = [float(sum(sorted(s[i * size:(i + 1) * size].tolist(), reverse=True)[:2])) for i in range(n)]
    open_groups = sorted(range(n), key=lambda i: (-total[i], i))[:router["groups"]["keep"]]
    allowed = [e for e in range(E) if e // size in open_groups]
    chosen = sorted(allowed, key=lambda e: (-float(s[e]), e))[:router["top"]]
    norm = sum(s[e] for e in chosen) + 1e-20
    return {e: s[e] / norm * router["scale"] for e in chosen}


def moe(h, w, p, f):
    z = h @ w[p + ".router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in route(z[t], f["router"]).items():
            out[t] += c * square_relu_ffn(h[t], w, f"{p}.e{e}")
    if f.get("shared"):
        out = out + sigmoid(h @ w[p + ".shared.sg"].T) * square_relu_ffn(h, w, p + ".shared")
    return out


def feed_forward(h, w, p, f):
    return gated_ffn(h, w, p) if f["kind"] == "dense" else moe(h, w, p, f)


def runs(cfg):
    """(layer, whether it begins a pass of the loop) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)]
            + [(i, False) for i in range(b, n)])


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) collects the residual stream after each layer run."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = x0 = model_norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    for i, first in runs(cfg):
        if first:
            x = torch.cat([x, x0], 1) @ w["loop.in"].T
        p, layer = f"l{i}", cfg["layers"][i]
        mixer = {"attention": attention, "channel_delta": channel_delta}[layer["type"]]
        x = x + m * mixer(model_norm(x, w[p + ".norm1"], eps), w, p + ".mix", layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + m * feed_forward(model_norm(x, w[p + ".norm2"], eps), w, p + ".mlp", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x)
    return model_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
