"""Plain, slow implementation of the Pemezen design, one function per mechanism, written from its equations.

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


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, w, groups, eps):
    """RMS norm of each of ``groups`` equal consecutive parts, times w."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * w


def short_conv(x, taps, bias=None):
    """Causal depth-wise convolution; the last column of ``taps`` weighs the current token; x [T, channels]."""
    K = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y if bias is None else y + bias


def input_conv(n, taps):
    return n + short_conv(n, taps)


def frequencies(rot):
    """(rotation frequency per pair, factor of cos and sin)."""
    d, base, s = rot["dims"], rot["base"], rot["scaling"]
    where = lambda turns: d * math.log(s["original"] / (turns * 2 * math.pi)) / (2 * math.log(base))      # noqa: E731
    lo = max(math.floor(where(s["fast"])), 0)
    hi = min(math.ceil(where(s["slow"])), d - 1)
    out = []
    for i in range(d // 2):
        f = base ** (-2 * i / d)
        r = min(max((i - lo) / max(hi - lo, 1e-3), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, positions, rot):
    """x [T, ..., >= dims]: neighbouring pairs of the first ``dims`` dimensions turn with the position."""
    f, m = frequencies(rot)
    angle = torch.as_tensor(list(positions), dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    c, s = torch.cos(angle) * m, torch.sin(angle) * m
    y = x.clone()
    for i in range(len(f)):
        u, v = x[..., 2 * i].transpose(0, -1), x[..., 2 * i + 1].transpose(0, -1)   # tokens last
        y[..., 2 * i] = (u * c[:, i] - v * s[:, i]).transpose(0, -1)
        y[..., 2 * i + 1] = (v * c[:, i] + u * s[:, i]).transpose(0, -1)
    return y


def latent_heads(q, c, kr, wuk, wuv, scale, dim):
    """q [Tq, H, dim + rot] of the last Tq positions (rotated), latents c [T, rank], shared rotated key part kr [T, rot]:
    softmax(scores) values per head, [Tq, H, vdim]."""
    Tq, H, T = q.shape[0], q.shape[1], c.shape[0]
    out = []
    for h in range(H):
        k = c @ wuk.reshape(H, dim, -1)[h].T
        v = c @ wuv.reshape(H, -1, c.shape[1])[h].T
        s = (q[:, h, :dim] @ k.T + q[:, h, dim:] @ kr.T) * scale
        seen = torch.arange(T)[None, :] <= (torch.arange(T - Tq, T)[:, None])
        s = s.masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append((e / e.sum(-1, keepdim=True)) @ v)
    return torch.stack(out, 1)


def latent_attention(h, w, p, m, eps, per_head_gate):
    T, H, dim, rd, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    pos = range(T)
    q = (h @ w[p + ".q"].T).reshape(T, H, dim + rd).clone()
    q[..., dim:] = rotate(q[..., dim:], pos, m["rot"])
    ckr = h @ w[p + ".dkv"].T
    c = rms(ckr[:, :L], eps) * w[p + ".dkv.norm"]
    kr = rotate(ckr[:, L:], pos, m["rot"])
    o = latent_heads(q, c, kr, w[p + ".uk"], w[p + ".uv"], m["scale"], dim)
    g = sigmoid(h @ w[p + ".g"].T)
    o = o * (g[:, :, None] if per_head_gate else g.reshape(o.shape))
    return o.reshape(T, -1) @ w[p + ".o"].T


def block_product(u, blocks, bias):
    """u in equal parts, each times its own square matrix [out, in]; blocks [n, d, d], bias [n, d]."""
    n, d = bias.shape
    return (torch.einsum("tbi,boi->tbo", u.reshape(-1, n, d), blocks) + bias).reshape(u.shape)


def gated_recurrence(u, r, i, lam, S=None):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); returns (all S, last S)."""
    S = torch.zeros_like(u[0]) if S is None else S
    out = []
    for t in range(u.shape[0]):
        a = torch.exp(-8 * r[t] * softplus(lam))
        S = a * S + torch.sqrt(1 - a * a) * i[t] * u[t]
        out.append(S)
    return torch.stack(out), S


def rglru(h, w, p):
    y = gelu_tanh(h @ w[p + ".y"].T + w[p + ".y.b"])
    u = short_conv(h @ w[p + ".x"].T + w[p + ".x.b"], w[p + ".conv"], w[p + ".conv.b"])
    r = sigmoid(block_product(u, w[p + ".ra"], w[p + ".ra.b"]))
    i = sigmoid(block_product(u, w[p + ".ri"], w[p + ".ri.b"]))
    S, _ = gated_recurrence(u, r, i, w[p + ".lam"])
    return (S * y) @ w[p + ".o"].T


def xielu(z, p, q):
    neg = torch.clamp(z, max=0)
    return torch.where(z > 0, softplus(p) * z * z + z / 2, (0.5 + softplus(q)) * (torch.exp(neg) - 1 - neg) + z / 2)


def dense_ffn(h, w, p):
    return xielu(h @ w[p + ".up"].T, w[p + ".act"][0], w[p + ".act"][1]) @ w[p + ".down"].T


def mixer(kind, h, w, p, m, eps):
    if kind == "rglru":
        return rglru(h, w, p)
    return latent_attention(h, w, p, m, eps, per_head_gate=kind == "latent_attention_2")


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) collects the residual stream after each layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps, G = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        h = input_conv(group_norm(x, w[p + ".norm1"], G, eps), w[p + ".canon1"])
        x = x + group_norm(mixer(layer["type"], h, w, p + ".mix", layer["mixer"], eps), w[p + ".norm1b"], G, eps)
        if layer["mlp"] is not None:
            h = input_conv(group_norm(x, w[p + ".norm2"], G, eps), w[p + ".canon2"])
            x = x + group_norm(dense_ffn(h, w, p + ".mlp"), w[p + ".norm2b"], G, eps)
        if layers_out is not None:
            layers_out.append(x)
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(group_norm(x, w["final.norm"], G, eps) @ w["head"].T / cap)
