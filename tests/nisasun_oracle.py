"""Plain, slow implementation of the Nisasun design, one function per mechanism, written from its equations.

It shares no code with the product path: float64 (or the dtype of the inputs) tensor arithmetic, one sequence at a
time, one token at a time wherever a recurrence is involved. ``cfg`` is the raw ``config.json`` dictionary and ``w``
maps the checkpoint's tensor names to tensors.
"""
import math

import torch


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def stream_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def window_attention(h, w, p, spec, eps):
    """Grouped-query softmax attention without rotation over the last ``mask.size`` tokens; h [T, width]."""
    T = h.shape[0]
    H, G, dk, dv = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    W = spec["mask"]["size"]
    q = (h @ w[p + ".q"].T).view(T, H, dk)
    k = (h @ w[p + ".k"].T).view(T, G, dk)
    v = (h @ w[p + ".v"].T).view(T, G, dv)
    q = rms(q, eps) * w[p + ".q.norm"]
    k = rms(k, eps) * w[p + ".k.norm"]
    out = h.new_zeros(T, H, dv)
    for i in range(T):
        lo = max(0, i - W + 1)
        for n in range(H):
            g = n // (H // G)
            s = (k[lo:i + 1, g] @ q[i, n]) * spec["scale"]
            e = torch.exp(s - s.max())
            out[i, n] = (e / e.sum()) @ v[lo:i + 1, g]
    return out.reshape(T, H * dv) @ w[p + ".o"].T


def decayed_outer_products(q, k, v, decay, S=None):
    """S_t = decay_t S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head. q, k [T, heads, n]; v [T, heads, m]; decay
    [T, heads]. Returns (o [T, heads, m], final S [heads, n, m])."""
    T, H, n = k.shape
    m = v.shape[2]
    S = k.new_zeros(H, n, m) if S is None else S.clone()
    o = k.new_zeros(T, H, m)
    for t in range(T):
        for h in range(H):
            S[h] = decay[t, h] * S[h] + torch.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def lightning(h, w, p, spec, eps):
    T = h.shape[0]
    H, dk, dv = spec["heads"], spec["dim"], spec["vdim"]
    q = silu(h @ w[p + ".q"].T).view(T, H, dk)
    k = silu(h @ w[p + ".k"].T).view(T, H, dk)
    v = silu(h @ w[p + ".v"].T).view(T, H, dv)
    decay = torch.tensor(spec["decay"], dtype=h.dtype).expand(T, H)
    o, _ = decayed_outer_products(q, k, v, decay)
    o = rms(o.reshape(T, H * dv), eps) * w[p + ".norm"]
    return (o / (1 + torch.exp(-(h @ w[p + ".g"].T)))) @ w[p + ".o"].T


def short_conv(x, taps, bias):
    """Causal depth-wise convolution, the last column of ``taps`` weighs the current token; x [T, channels]."""
    K = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y + bias


def state_space(h, w, p, spec, eps):
    """Mamba-2: input projection, short convolution, scalar-decay state, skip, gate before a grouped norm."""
    T = h.shape[0]
    H, P, N, G = spec["heads"], spec["vdim"], spec["state"], spec["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w[p + ".in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(short_conv(xbc, w[p + ".conv"], w[p + ".conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    x, B, C = x.view(T, H, P), B.view(T, G, N), C.view(T, G, N)
    a = dt + w[p + ".dt_bias"]
    dt = torch.clamp(a, min=0) + torch.log1p(torch.exp(-a.abs()))
    group = [n // (H // G) for n in range(H)]
    decay = torch.exp(-torch.exp(w[p + ".A_log"]) * dt)
    y, _ = decayed_outer_products(C[:, group], B[:, group], x * dt[..., None], decay)
    y = y + w[p + ".D"][:, None] * x
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, spec["norm_groups"], -1), eps).reshape(T, inner) * w[p + ".norm"]
    return y @ w[p + ".o"].T


def parallel(h, w, p, spec, eps):
    return (spec["left_scale"] * window_attention(h, w, p + ".left", spec["left"], eps)
            + spec["right_scale"] * state_space(h, w, p + ".right", spec["right"], eps))


def dense_ffn(h, w, p):
    return (gelu_tanh(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def route(scores, correction, router):
    """Chosen expert ids of one token: scores and correction [experts]."""
    E, n_g = router["experts"], router["groups"]["count"]
    choice = (scores + correction).tolist()
    per = E // n_g
    best = sorted(range(n_g), key=lambda g: (-max(choice[g * per:(g + 1) * per]), g))[:router["groups"]["keep"]]
    open_ = [e for e in range(E) if e // per in best]
    return sorted(open_, key=lambda e: (-choice[e], e))[:router["top"]]


def moe_ffn(h, w, p, spec):
    r = spec["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        z = w[p + ".router"] @ h[t]
        e = torch.exp(z - z.max())
        s = e / e.sum()
        for x in route(s, w[p + ".correction"], r):
            q = f"{p}.e{x}"
            out[t] += s[x] * (w[q + ".down"] @ (silu(w[q + ".gate"] @ h[t]) * (w[q + ".up"] @ h[t])))
    return out


def hyper(X, w, name, norm_w, sublayer, eps):
    """One sublayer between hyper-connections: X [T, streams, width]."""
    u = torch.einsum("s,tsd->td", w[name + ".in"], X)
    y = sublayer(stream_norm(u, norm_w, eps))
    return torch.einsum("st,nsd->ntd", w[name + ".mix"], X) + w[name + ".out"][None, :, None] * y[:, None, :]


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` (a list) collects the sum of the streams after each layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = torch.stack([x] * cfg["streams"], 1)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        mixer = {"lightning": lightning, "parallel": parallel}[layer["type"]]
        X = hyper(X, w, p + ".hc1", w[p + ".norm1"], lambda h: mixer(h, w, p + ".mix", layer["mixer"], eps), eps)
        ff = layer["mlp"]
        if ff is not None:
            f = (lambda h: dense_ffn(h, w, p + ".mlp")) if ff["kind"] == "dense" else (lambda h: moe_ffn(h, w, p + ".mlp", ff))
            X = hyper(X, w, p + ".hc2", w[p + ".norm2"], f, eps)
        if layers_out is not None:
            layers_out.append(X.sum(1))
    return stream_norm(X.sum(1), w["final.norm"], eps) @ w["head"].T
