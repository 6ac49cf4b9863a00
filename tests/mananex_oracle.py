"""Plain, slow implementation of the Mananex design, one function per mechanism, written from its equations.

It shares no code with the product path: float64 (or the dtype of the inputs) tensor arithmetic, one sequence at a time,
one token at a time wherever a recurrence is involved. ``cfg`` is the raw ``config.json`` dictionary and ``w`` maps the
checkpoint's tensor names to tensors.
"""
import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def model_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def rotate(x, positions, rot):
    """x [T, heads, >= dims]: columns 2i and 2i + 1 turn by the position times base^(-2i / dims)."""
    y = x.clone()
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        for t, p in enumerate(positions):
            c, s = math.cos(p * f), math.sin(p * f)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i], y[t, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def sees(i, j, mask):
    """Whether position i attends to position j: causal, inside the window or one of the kept first tokens."""
    return j <= i and (i - j < mask["size"] or j < mask["keep_first"])


def sink_softmax(q, k, v, scale, mask, sink):
    """q [Tq, H, d] of the last Tq of T positions, k [T, G, d], v [T, G, dv], sink [H]: [Tq, H, dv]. The sink adds
    exp(sink) to the denominator."""
    Tq, H, T, G = q.shape[0], q.shape[1], k.shape[0], k.shape[1]
    ok = torch.tensor([[sees(i, j, mask) for j in range(T)] for i in range(T - Tq, T)])
    out = []
    for h in range(H):
        s = ((q[:, h] @ k[:, h // (H // G)].T) * scale).masked_fill(~ok, -math.inf)
        top = torch.maximum(s.max(-1, keepdim=True).values, sink[h])
        e = torch.exp(s - top)
        out.append((e / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - top))) @ v[:, h // (H // G)])
    return torch.stack(out, 1)


def attention(h, w, p, m):
    """The left mixer: rotated, windowed grouped-query attention with a sink and a gate per head."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rotate((h @ w[p + ".q"].T).reshape(T, H, m["dim"]), range(T), m["rot"])
    k = rotate((h @ w[p + ".k"].T).reshape(T, G, m["dim"]), range(T), m["rot"])
    v = (h @ w[p + ".v"].T).reshape(T, G, m["vdim"])
    o = sink_softmax(q, k, v, m["scale"], m["mask"], w[p + ".sink"])
    o = o * sigmoid(h @ w[p + ".g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + ".o"].T


def forget(z, lower):
    """Forget gate held above ``lower``."""
    return lower + (1 - lower) * sigmoid(z)


def forget_write(q, f, v, S=None):
    """q, f [T, H, d], v [T, H, dv]: each row of the state keeps f of itself and takes 1 - f of the value. Returns
    (o [T, H, dv], last S [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def hgrn2(h, w, p, m, eps):
    """The right mixer: a matrix state whose forget gate also decides what is written, a norm per head behind it."""
    T, H = h.shape[0], m["heads"]
    q = silu(h @ w[p + ".q"].T).reshape(T, H, m["dim"])
    f = forget(h @ w[p + ".f"].T + w[p + ".f.b"], w[p + ".lower"]).reshape(T, H, m["dim"])
    v = (h @ w[p + ".v"].T).reshape(T, H, m["vdim"])
    o, _ = forget_write(q, f, v)
    return (rms(o, eps) * w[p + ".norm"]).reshape(T, -1) @ w[p + ".o"].T


def parallel(h, w, p, m, eps):
    return m["left_scale"] * attention(h, w, p + ".left", m["left"]) + m["right_scale"] * hgrn2(h, w, p + ".right", m["right"], eps)


def gated_ffn(h, w, p, bias):
    lin = lambda x, n: x @ w[f"{p}.{n}"].T + (w[f"{p}.{n}.b"] if bias else 0)     # noqa: E731
    return lin(silu(lin(h, "gate")) * lin(h, "up"), "down")


def route(z, top):
    """Logits z [experts] of one token -> {expert: weight}: the largest ``top``, softmax over those."""
    chosen = sorted(range(z.shape[0]), key=lambda e: (-float(z[e]), e))[:top]
    e = torch.exp(z[chosen] - z[chosen].max())
    return dict(zip(chosen, e / e.sum()))


def moe(h, w, p, f):
    z = h @ w[p + ".router"].T + w[p + ".router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in route(z[t], f["router"]["top"]).items():
            out[t] += c * gated_ffn(h[t], w, f"{p}.e{e}", False)
    return out


def feed_forward(h, w, p, f):
    return gated_ffn(h, w, p, True) if f["kind"] == "dense" else moe(h, w, p, f)


def depth_average(coef, outputs):
    """Weighted sum of the embedding output and every layer's result so far."""
    x = torch.zeros_like(outputs[0])
    for c, o in zip(coef, outputs, strict=True):
        x = x + c * o
    return x


def layer(x, w, p, spec, eps):
    """One norm, both sublayers on its output, each gated element by element on the way into the residual."""
    h = model_norm(x, w[p + ".norm1"], eps)
    gate = lambda n: sigmoid(h @ w[f"{p}.{n}"].T + w[f"{p}.{n}.b"])               # noqa: E731
    y = gate("rg1") * parallel(h, w, p + ".mix", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        y = y + gate("rg2") * feed_forward(h, w, p + ".mlp", spec["mlp"])
    return x + y


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) collects what each layer hands to the next."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    outputs = [x]
    for i, spec in enumerate(cfg["layers"]):
        outputs.append(layer(x, w, f"l{i}", spec, eps))
        x = depth_average(w[f"l{i}.dwa"], outputs)
        if layers_out is not None:
            layers_out.append(x)
    return model_norm(x, w["final.norm"], eps) @ w["embed"].T
