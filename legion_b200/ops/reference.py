"""Plain PyTorch reference of every op (the oracle for the sm_100a kernels and the CPU back-end).

All math is done in float32 whatever the input dtype; outputs are cast back to the input dtype.
Shapes follow the kernel interfaces: activations are token-major ``[T, features]``, the paged KV
cache is ``[blocks, page, kv_heads, head_dim]`` and a block table row lists a sequence's blocks.
Reference counterparts: the CPU implementation of each external op in the reference engine
(``src/model/core/*.rs`` ``cpu`` functions, e.g. ``src/model/core/gdn_scan.rs:195-262``).
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn.functional as F


def rmsnorm(x, w, eps: float, w_offset: float = 0.0, residual=None):
    """Returns (normed, summed) where summed = x (+ residual)."""
    xf = x.float()
    if residual is not None:
        xf = (xf + residual.float()).to(x.dtype).float()
    summed = xf.to(x.dtype)
    inv = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    y = xf * inv * (w.float() + w_offset)
    return y.to(x.dtype), summed


def linear(x, w, residual=None, out_dtype=None):
    y = x.float() @ w.float().t()
    if residual is not None:
        y = y + residual.float()
    return y.to(out_dtype or x.dtype)


def gate_up_act(x, w_gate_up, n_ff: int, act: str = "silu", bias=None):
    """w_gate_up rows: [gate(n_ff) | up(n_ff)]; returns act(gate) * up."""
    h = x.float() @ w_gate_up.float().t()
    if bias is not None:
        h = h + bias
    if w_gate_up.shape[0] == n_ff:            # un-gated FFN (squared ReLU): only the up projection exists
        return activation(h, act).to(x.dtype)
    g, u = h[:, :n_ff], h[:, n_ff:2 * n_ff]
    return (activation(g, act) * u).to(x.dtype)


def activation(g, act: str):
    if act == "silu":
        return F.silu(g)
    if act == "gelu_tanh":
        return F.gelu(g, approximate="tanh")
    if act == "relu2":
        return F.relu(g).pow(2)
    raise ValueError(act)


def rope_cos_sin(max_pos: int, rot: int, theta: float, scaling: Optional[dict] = None, device="cpu"):
    """Table [max_pos, rot] = [cos(rot/2) | sin(rot/2)] in float32."""
    half = rot // 2
    inv_freq = 1.0 / (theta ** (torch.arange(0, half, dtype=torch.float64, device=device) / half))
    mag = 1.0
    if scaling:
        kind = scaling.get("type", scaling.get("rope_type", "linear"))
        factor = float(scaling.get("factor", 1.0))
        if kind == "linear":
            inv_freq = inv_freq / factor
        elif kind == "factors":           # per-frequency divisors (a checkpoint's ``rope_freqs`` tensor)
            inv_freq = inv_freq / torch.tensor(scaling["factors"], dtype=torch.float64, device=device)
        elif kind == "llama3":
            low = float(scaling.get("low_freq_factor", 1.0))
            high = float(scaling.get("high_freq_factor", 4.0))
            orig = float(scaling.get("original_max_position_embeddings", 8192))
            wavelen = 2 * math.pi / inv_freq
            smooth = (orig / wavelen - low) / (high - low)
            scaled = torch.where(wavelen > orig / low, inv_freq / factor, inv_freq)
            mid = (1 - smooth) * inv_freq / factor + smooth * inv_freq
            is_mid = (wavelen <= orig / low) & (wavelen >= orig / high)
            inv_freq = torch.where(is_mid, mid, scaled)
        elif kind == "yarn":
            # NTK-by-parts: high-frequency pairs keep their wavelength, low-frequency pairs are interpolated by
            # ``factor``, a linear ramp between the pairs that turn beta_fast and beta_slow times over the original
            # context; cos and sin carry the attention factor (0.1 ln(factor) + 1 unless the checkpoint gives one,
            # or the ratio of its two mscale terms)
            orig = float(scaling.get("original_max_position_embeddings") or max_pos)
            fast, slow = float(scaling.get("beta_fast") or 32.0), float(scaling.get("beta_slow") or 1.0)

            def corr(n_rot):
                return rot * math.log(orig / (n_rot * 2 * math.pi)) / (2 * math.log(theta))

            lo, hi = corr(fast), corr(slow)
            if scaling.get("truncate", True):
                lo, hi = math.floor(lo), math.ceil(hi)
            lo, hi = max(lo, 0), min(hi, rot - 1)
            ramp = ((torch.arange(half, dtype=torch.float64, device=device) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
            inv_freq = inv_freq / factor * ramp + inv_freq * (1 - ramp)
            mag = yarn_attention_factor(scaling)
    pos = torch.arange(max_pos, dtype=torch.float64, device=device)
    ang = pos[:, None] * inv_freq[None, :]
    return (torch.cat([ang.cos(), ang.sin()], dim=-1) * mag).float()


def yarn_mscale(factor: float, m: float = 1.0) -> float:
    return 1.0 if factor <= 1 else 0.1 * m * math.log(factor) + 1.0


def yarn_attention_factor(scaling: dict) -> float:
    """What YaRN multiplies cos and sin with (so attention scores grow by its square)."""
    if scaling.get("attention_factor") is not None:
        return float(scaling["attention_factor"])
    factor = float(scaling.get("factor", 1.0))
    m, m_all = scaling.get("mscale"), scaling.get("mscale_all_dim")
    if m and m_all:
        return yarn_mscale(factor, float(m)) / yarn_mscale(factor, float(m_all))
    return yarn_mscale(factor)


def apply_rope(x, cos_sin, positions, rot: int):
    """x: [T, H, D]; rotate-half pairing (i, i + rot/2) over the first ``rot`` dims."""
    if rot <= 0:
        return x
    half = rot // 2
    cs = cos_sin[positions.long()]
    c, s = cs[:, None, :half], cs[:, None, half:rot]
    xf = x.float()
    a, b = xf[..., :half], xf[..., half:rot]
    out = xf.clone()
    out[..., :half] = a * c - b * s
    out[..., half:rot] = b * c + a * s
    return out.to(x.dtype)


def head_rmsnorm(x, w, eps, w_offset=0.0):
    xf = x.float()
    inv = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (xf * inv * (w.float() + w_offset)).to(x.dtype)


def qk_norm_rope_append(qkv, n_q, n_kv, d, q_norm_w, k_norm_w, eps, w_offset, cos_sin, rot, positions, slots,
                        k_cache, v_cache, gated_q: bool = False):
    """Splits the fused projection, norms + ropes q and k, appends k, v to the paged cache in place.

    With ``gated_q`` the q block is laid out per head as [q(d) | gate(d)]. Returns (q [T, n_q, d], gate or None).
    """
    T = qkv.shape[0]
    qw = n_q * d * (2 if gated_q else 1)
    qpart = qkv[:, :qw].reshape(T, n_q, -1)
    gate = qpart[..., d:] if gated_q else None
    q = qpart[..., :d]
    k = qkv[:, qw:qw + n_kv * d].reshape(T, n_kv, d)
    v = qkv[:, qw + n_kv * d:qw + 2 * n_kv * d].reshape(T, n_kv, d)
    if q_norm_w is not None:
        q = head_rmsnorm(q, q_norm_w, eps, w_offset)
    if k_norm_w is not None:
        k = head_rmsnorm(k, k_norm_w, eps, w_offset)
    q = apply_rope(q, cos_sin, positions, rot)
    k = apply_rope(k, cos_sin, positions, rot)
    page = k_cache.shape[1]
    valid = slots >= 0
    sl = slots[valid].long()
    k_cache.view(-1, n_kv, d)[sl] = k[valid].to(k_cache.dtype)
    v_cache.view(-1, n_kv, d)[sl] = v[valid].to(v_cache.dtype)
    _ = page
    return q.contiguous(), gate


def _gather_kv(cache, table_row, n_tokens):
    page = cache.shape[1]
    n_blocks = (n_tokens + page - 1) // page
    blocks = table_row[:n_blocks].long()
    return cache[blocks].reshape(-1, cache.shape[2], cache.shape[3])[:n_tokens]


def paged_attention(q, k_cache, v_cache, block_table, ctx_lens, cu_q, scale, window: int = 0, causal: bool = True,
                    sinks=None, softcap: float = 0.0, keep_first: int = 0, gate=None, out_scale: float = 1.0):
    """Varlen paged attention. q: [T, Hq, D]; sequence i owns query rows cu_q[i]:cu_q[i+1], which are the
    LAST rows of its ctx_lens[i] cached tokens. Returns [T, Hq, Dv] (values may have a head size of their own).
    ``keep_first``: first tokens that a window leaves visible; ``sinks`` [Hq]: exp(sink) joins the denominator; the output
    times ``out_scale`` and, with ``gate`` [T, Hq], times its sigmoid."""
    T, Hq, D = q.shape
    Hkv = k_cache.shape[2]
    G = Hq // Hkv
    out = q.new_zeros(T, Hq, v_cache.shape[3])
    for i in range(len(ctx_lens)):
        q0, q1 = int(cu_q[i]), int(cu_q[i + 1])
        if q1 <= q0:
            continue
        ctx = int(ctx_lens[i])
        k = _gather_kv(k_cache, block_table[i], ctx).float()
        v = _gather_kv(v_cache, block_table[i], ctx).float()
        qi = q[q0:q1].float()
        k = k.repeat_interleave(G, dim=1)
        v = v.repeat_interleave(G, dim=1)
        s = torch.einsum("qhd,khd->hqk", qi, k) * scale
        if softcap > 0:
            s = torch.tanh(s / softcap) * softcap
        qpos = torch.arange(ctx - (q1 - q0), ctx, device=q.device)[:, None]
        kpos = torch.arange(ctx, device=q.device)[None, :]
        mask = torch.ones(q1 - q0, ctx, dtype=torch.bool, device=q.device)
        if causal:
            mask &= kpos <= qpos
        if window > 0:
            mask &= (kpos > qpos - window) | (kpos < keep_first)
        s = s.masked_fill(~mask[None], float("-inf"))
        if sinks is not None:
            s = torch.cat([s, sinks.float().view(Hq, 1, 1).expand(Hq, q1 - q0, 1)], dim=-1)
            p = torch.softmax(s, dim=-1)[..., :-1]
        else:
            p = torch.softmax(s, dim=-1)
        p = torch.nan_to_num(p)
        o = torch.einsum("hqk,khd->qhd", p, v) * out_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[q0:q1].float()).unsqueeze(2)
        out[q0:q1] = o.to(q.dtype)
    return out


def router_topk(logits, k: int, mode: str = "softmax", renorm: bool = True, route_scale: float = 1.0, bias=None,
                n_group: int = 1, topk_group: int = 1, group_top: int = 2):
    """Returns (ids [T, k] int32, weights [T, k] float32); ties go to the lower expert id. ``renorm``: True holds the sum
    of the chosen weights away from zero, "sum" divides by it as it is. ``biased_softmax``: the bias joins the logits;
    ``softmax_bias``: selection
    by softmax score + bias, like the sigmoid mode; ``group_top``: how many scores a group's rank sums up."""
    lf = logits.float()
    T, E = lf.shape
    if mode in ("softmax", "biased_softmax"):
        scores = torch.softmax(lf if mode == "softmax" else lf + bias.float(), dim=-1)
        sel = scores.clone()
    else:
        scores = torch.softmax(lf, dim=-1) if mode == "softmax_bias" else torch.sigmoid(lf)
        sel = scores + (bias.float() if bias is not None else 0.0)
        if n_group > 1 and topk_group < n_group:
            g = sel.view(T, n_group, E // n_group)
            gscore = g.topk(min(group_top, g.shape[-1]), dim=-1).values.sum(-1)
            order = torch.sort(gscore, dim=-1, descending=True, stable=True).indices[:, :topk_group]
            keep = torch.zeros(T, n_group, dtype=torch.bool, device=lf.device)
            keep.scatter_(1, order, True)
            sel = g.masked_fill(~keep[:, :, None], float("-inf")).reshape(T, E)
    order = torch.sort(sel, dim=-1, descending=True, stable=True).indices[:, :k]
    w = scores.gather(1, order)
    if renorm == "sum":
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    elif renorm:
        w = w / w.sum(-1, keepdim=True).clamp_min(6.1e-5)
    return order.int(), (w * route_scale).float()


def moe_experts(x, ids, wts, w_gate_up, w_down, n_ff: int, act: str = "silu", e_lo: int = 0, e_hi: Optional[int] = None):
    """Routed expert FFN. w_gate_up: [E, 2*n_ff, H] ([gate | up] rows), w_down: [E, H, n_ff].
    Only experts in [e_lo, e_hi) contribute (expert parallel shards). Returns float32 [T, H]."""
    T, H = x.shape
    E = w_gate_up.shape[0]
    e_hi = E + e_lo if e_hi is None else e_hi
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    xf = x.float()
    for e in range(e_lo, e_hi):
        hit = ids == e
        if not bool(hit.any()):
            continue
        tok, choice = hit.nonzero(as_tuple=True)
        le = e - e_lo
        h = xf[tok] @ w_gate_up[le].float().t()
        if h.shape[1] == n_ff:            # un-gated experts (squared ReLU): one up projection
            h = activation(h, act).to(x.dtype).float()
        else:
            h = (activation(h[:, :n_ff], act) * h[:, n_ff:]).to(x.dtype).float()
        y = (h @ w_down[le].float().t()) * wts[tok, choice][:, None]
        out.index_add_(0, tok, y.to(x.dtype).float())
    return out


def argmax(logits):
    return torch.argmax(logits.float(), dim=-1).int()


def causal_conv1d_silu(x, w, bias, conv_state, cu_seq, slots, write_state: bool = True, in_bias=None, silu: bool = True):
    """x: [T, C]; w: [C, KC]; conv_state: [slots, C, KC-1] float32 (oldest first). ``in_bias`` is added to x first (the
    history holds the sums; before a sequence's start there is zero)."""
    out = torch.empty_like(x)
    KC = w.shape[1]
    for i in range(len(slots)):
        t0, t1 = int(cu_seq[i]), int(cu_seq[i + 1])
        if t1 <= t0:
            continue
        s = int(slots[i])
        hist = conv_state[s].float().t()  # [KC-1, C]
        rows = x[t0:t1].float() if in_bias is None else x[t0:t1].float() + in_bias.float()
        seq = torch.cat([hist, rows], dim=0)
        win = seq.unfold(0, KC, 1)  # [n, C, KC]
        y = (win * w.float()[None]).sum(-1)
        if bias is not None:
            y = y + bias.float()
        out[t0:t1] = (F.silu(y) if silu else y).to(x.dtype)
        if write_state and KC > 1:
            conv_state[s] = seq[-(KC - 1):].t().to(conv_state.dtype)
    return out


def qkv_conv_append(proj, in_b, conv_w, conv_state, cu_seq, state_slots, q_norm, k_norm, norm_over, eps, rot, layout,
                    positions, slots, k_cache, v_cache, heads: int, write_state: bool = True):
    """``proj`` [T, q | k | v]: bias, short convolution (conv_w [taps, columns]) with carried history [slots, taps - 1, columns], norm of q and k over each head or the whole,
    rotation, k and v to their cache cells. Everything behind the projection is optional (None). Returns q [T, heads, dk]
    in the activation type; the values between are float32."""
    n_kv, dk, dv = k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    T, nq, nk = proj.shape[0], heads * dk, n_kv * dk
    u = proj.float() if in_b is None else proj.float() + in_b
    if conv_w is not None and conv_w.shape[0] == 1:
        u = u * conv_w[0]
    elif conv_w is not None:
        u = causal_conv1d_silu(u, conv_w.t(), None, conv_state.transpose(1, 2), cu_seq, state_slots, write_state, None, False)
    q, k, v = u[:, :nq], u[:, nq:nq + nk], u[:, nq + nk:nq + nk + n_kv * dv]
    if q_norm is not None and norm_over == "all":
        q, k = _norm32(q, q_norm, eps, 0.0), _norm32(k, k_norm, eps, 0.0)
    q, k = q.reshape(T, heads, dk), k.reshape(T, n_kv, dk)
    if q_norm is not None and norm_over == "head":
        q, k = _norm32(q, q_norm, eps, 0.0), _norm32(k, k_norm, eps, 0.0)
    if rot is not None:
        turn = rotate_pairs if layout == "pairs" else (lambda x, cs, p: apply_rope(x, cs, p, cs.shape[1]))
        q, k = turn(q, rot, positions), turn(k, rot, positions)
    ok = slots >= 0
    k_cache.view(-1, n_kv, dk)[slots[ok].long()] = k[ok].to(k_cache.dtype)
    v_cache.view(-1, n_kv, dv)[slots[ok].long()] = v.reshape(T, n_kv, dv)[ok].to(v_cache.dtype)
    return q.to(proj.dtype).contiguous()


def channel_delta(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H: int, G: int, dk: int, dv: int,
                  write_state: bool = True):
    """Gated delta rule with a decay per key channel. ``qkv`` [T, q | k | v] in front of the short convolution (conv_w
    [taps, columns], history [slots, taps - 1, columns]), ``a_raw``
    [T, H * dk] and ``b_raw`` [T, H] before their activations, state [slots, H, dv, dk] float32. Per head
    S = g S (key channels), S += k (beta (v - S^T k))^T, o = S^T q. Returns o [T, H * dv]."""
    T = qkv.shape[0]
    u = causal_conv1d_silu(qkv, conv_w.t(), None, conv_state.transpose(1, 2), cu_seq, slots, write_state).float()
    unit = lambda x: x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)                  # noqa: E731
    q = unit(u[:, :G * dk].reshape(T, G, dk)).repeat_interleave(H // G, 1) * dk ** -0.5
    k = unit(u[:, G * dk:2 * G * dk].reshape(T, G, dk)).repeat_interleave(H // G, 1)
    v = u[:, 2 * G * dk:].reshape(T, H, dv)
    g = torch.exp(A.float()[:, None] * F.softplus(a_raw.float() + dt_bias).view(T, H, dk))
    beta = torch.sigmoid(b_raw.float())
    out = torch.empty(T, H, dv, dtype=torch.float32, device=qkv.device)
    for i in range(len(slots)):
        S = state[int(slots[i])].clone()
        for t in range(int(cu_seq[i]), int(cu_seq[i + 1])):
            S = S * g[t].unsqueeze(1)
            d = beta[t].unsqueeze(1) * (v[t] - torch.einsum("hvk,hk->hv", S, k[t]))
            S = S + d.unsqueeze(2) * k[t].unsqueeze(1)
            out[t] = torch.einsum("hvk,hk->hv", S, q[t])
        if write_state:
            state[int(slots[i])] = S
    return out.reshape(T, H * dv).to(qkv.dtype)


def gdn_gates(a, b, A, dt_bias):
    g = A.float() * F.softplus(a.float() + dt_bias.float())
    return g, torch.sigmoid(b.float())


def gdn_recurrent(qkv, g, beta, state, cu_seq, slots, n_k, n_v, dk, dv, tiled_heads: bool, scale: float,
                  l2_eps: float = 1e-6, write_state: bool = True):
    """Gated delta rule, token by token. qkv: [T, 2*n_k*dk + n_v*dv]; state: [slots, n_v, dk, dv] float32."""
    T = qkv.shape[0]
    out = torch.zeros(T, n_v, dv, dtype=qkv.dtype, device=qkv.device)
    q_all = qkv[:, :n_k * dk].float().view(T, n_k, dk)
    k_all = qkv[:, n_k * dk:2 * n_k * dk].float().view(T, n_k, dk)
    v_all = qkv[:, 2 * n_k * dk:].float().view(T, n_v, dv)
    q_all = q_all * torch.rsqrt(q_all.pow(2).sum(-1, keepdim=True) + l2_eps) * scale
    k_all = k_all * torch.rsqrt(k_all.pow(2).sum(-1, keepdim=True) + l2_eps)
    heads = torch.arange(n_v, device=qkv.device)
    kh = heads % n_k if tiled_heads else heads // (n_v // n_k)
    for i in range(len(slots)):
        t0, t1 = int(cu_seq[i]), int(cu_seq[i + 1])
        s = int(slots[i])
        S = state[s].float().clone()  # [n_v, dk, dv]
        for t in range(t0, t1):
            q, k, v = q_all[t, kh], k_all[t, kh], v_all[t]
            gt = torch.exp(g[t].float())[:, None]
            bt = beta[t].float()[:, None]
            kv = torch.einsum("hkv,hk->hv", S, k)
            delta = (v - gt * kv) * bt
            S = gt[:, :, None] * S + k[:, :, None] * delta[:, None, :]
            out[t] = torch.einsum("hkv,hk->hv", S, q).to(out.dtype)
        if write_state:
            state[s] = S.to(state.dtype)
    return out


def gated_rmsnorm(o, z, w, eps: float, act: str = "silu"):
    """o, z: [T, H, D]; w: [D]."""
    of = o.float()
    y = of * torch.rsqrt(of.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    zf = z.float()
    return (y * (F.silu(zf) if act == "silu" else torch.sigmoid(zf))).to(o.dtype)


def hyper_start(rows, streams: int, in_w, norm_w, eps: float, w_offset: float):
    """Every stream starts as the embedding row. Returns (streams [T, S, H] float32, h = norm of the mixed input)."""
    X = rows.float().unsqueeze(1).expand(-1, streams, -1).contiguous()
    u = torch.einsum("s,tsh->th", in_w, X) if in_w is not None else X.sum(1)
    return X, _norm32(u, norm_w, eps, w_offset).to(rows.dtype)


def _norm32(u, w, eps, w_offset):
    return u / torch.sqrt(u.pow(2).mean(-1, keepdim=True) + eps) * (w.float() + w_offset)


def hyper_step(X, terms, mix, out_w, in_w, norm_w, eps: float, w_offset: float):
    """Static hyper-connection around a sublayer: y = sum of scale * tensor over ``terms``; X'_t = sum_s mix[s, t] X_s +
    out[t] y; returns (X', norm of the next sublayer's input sum_t in[t] X'_t). ``in_w`` None: plain sum."""
    y = sum(c * t.float() for t, c in terms)
    Xn = torch.einsum("st,nsh->nth", mix, X) + out_w[None, :, None] * y.unsqueeze(1)
    u = torch.einsum("s,tsh->th", in_w, Xn) if in_w is not None else Xn.sum(1)
    return Xn, _norm32(u, norm_w, eps, w_offset).to(terms[0][0].dtype)


def qkv_norm_append(q, k, v, q_norm, k_norm, eps, slots, k_cache, v_cache):
    """Head norms and paged append with separate key / value head sizes; returns q [T, Hq, dk]."""
    n_kv, dk, dv = k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    T = q.shape[0]
    q, k = q.reshape(T, -1, dk), k.reshape(T, n_kv, dk)
    if q_norm is not None:
        q, k = head_rmsnorm(q, q_norm, eps), head_rmsnorm(k, k_norm, eps)
    ok = slots >= 0
    k_cache.view(-1, n_kv, dk)[slots[ok].long()] = k[ok].to(k_cache.dtype)
    v_cache.view(-1, n_kv, dv)[slots[ok].long()] = v.reshape(T, n_kv, dv)[ok].to(v_cache.dtype)
    return q.contiguous()


def linear_scan(q, k, v, state, cu_seq, slots, H: int, G: int, N: int, P: int, decay=None, silu_in: bool = False,
                dt=None, dt_bias=None, A=None, D=None, z=None, write_state: bool = True):
    """S_t = a_t S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, token by token; state [slots, H, P, N] float32. ``decay`` [H]:
    constant per head; else a_t = exp(dt_t A) with dt_t = softplus(dt + dt_bias), which also scales v. D: skip; z: gate
    by silu(z). q, k [T, G * N], v [T, H * P]."""
    T = q.shape[0]
    qf, kf, vf = q.float().view(T, G, N), k.float().view(T, G, N), v.float().view(T, H, P)
    if silu_in:
        qf, kf, vf = F.silu(qf), F.silu(kf), F.silu(vf)
    qf, kf = qf.repeat_interleave(H // G, 1), kf.repeat_interleave(H // G, 1)
    if decay is not None:
        a, vd = decay.float().expand(T, H), vf
    else:
        step = F.softplus(dt.float() + dt_bias.float())
        a, vd = torch.exp(step * A.float()), vf * step.unsqueeze(-1)
    out = torch.zeros(T, H, P)
    for i in range(len(slots)):
        t0, t1, s = int(cu_seq[i]), int(cu_seq[i + 1]), int(slots[i])
        if t1 <= t0:
            continue
        S = state[s].clone()
        for t in range(t0, t1):
            S = S * a[t][:, None, None] + vd[t].unsqueeze(2) * kf[t].unsqueeze(1)
            out[t] = torch.einsum("hpn,hn->hp", S, qf[t])
        if write_state:
            state[s] = S
    if D is not None:
        out = out + D.float()[:, None] * vf
    out = out.reshape(T, H * P)
    if z is not None:
        out = out * F.silu(z.float())
    return out.to(q.dtype)


def group_norm_gate(y, gate, w, eps: float, groups: int = 1):
    """RMS norm in ``groups`` equal parts, times w, times sigmoid(gate) when given."""
    T, C = y.shape
    yf = y.float().view(T, groups, C // groups)
    out = (yf / torch.sqrt(yf.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, C) * w.float()
    if gate is not None:
        out = out * torch.sigmoid(gate.float())
    return out.to(y.dtype)


def prenorm_start(rows, pre_w, norm_w, eps: float, w_offset: float):
    """x [T, H] float32: the rows, normed with ``pre_w`` when given; and its norm (``norm_w`` None: none)."""
    x = rows.float() if pre_w is None else _norm32(rows.float(), pre_w, eps, w_offset)
    return x, None if norm_w is None else _norm32(x, norm_w, eps, w_offset).to(rows.dtype)


def prenorm_step(x, terms, mult: float, norm_w, eps: float, w_offset: float, dtype):
    """x + mult * (sum of scale * tensor over ``terms``) and the norm of that (``norm_w`` None: none)."""
    if terms:
        x = x + mult * sum(c * t.float() for t, c in terms)
    return x, None if norm_w is None else _norm32(x, norm_w, eps, w_offset).to(dtype)


def depth_step(x, hist, i: int, y1, g1, b1, y2, g2, b2, y2_b, coefs, norm_w, eps: float, w_offset: float, rows=None):
    """Behind layer ``i`` of a stack with parallel sublayers: X = x + sigmoid(g1 + b1) y1 + sigmoid(g2 + b2) (y2 + y2_b) (no
    gate without ``g1``; ``y2`` may be None). With ``hist`` (``hist.X`` [layers + 1, T, H] float32: the embedding output and the
    layers' results) X becomes its entry i + 1 and the next input is the sum of coefs[0][j] * hist.X[j] for j = 0 .. i + 1
    (``coefs``: of layer i, then of the layers behind it). Returns that and its norm, of the given ``rows`` only when there are
    any."""
    open_ = lambda g, b: 1.0 if g is None else torch.sigmoid(g.float() + b)                # noqa: E731
    X = x + open_(g1, b1) * y1.float()
    if y2 is not None:
        f = y2.float() if y2_b is None else y2.float() + y2_b
        X = X + open_(g2, b2) * f
    if hist is not None:
        hist.X[i + 1] = X
        X = torch.einsum("j,jth->th", coefs[0], hist.X[:i + 2])
    if rows is not None:
        X = X.index_select(0, rows)
    return X, _norm32(X, norm_w, eps, w_offset).to(y1.dtype)


def forget_scan(q, f, v, f_b, lower, state, cu_seq, slots, H: int, N: int, P: int, norm_w, eps: float, scale: float = 1.0,
                write_state: bool = True):
    """HGRN2: with F = lower + (1 - lower) sigmoid(f + f_b) per key channel, S_t = diag(F_t) S_(t-1) + (1 - F_t) v_t^T and
    o_t = S_t^T silu(q_t); q, f [T, H * N], v [T, H * P], state [slots, H, P, N] float32. Returns the RMS norm of each
    head's o times norm_w [P] times ``scale``, [T, H * P]."""
    T = q.shape[0]
    z = f.float() + f_b
    keep = (lower + (1 - lower) * torch.sigmoid(z)).view(T, H, N)
    write = ((1 - lower) * torch.sigmoid(-z)).view(T, H, N)
    qf, vf = F.silu(q.float()).view(T, H, N), v.float().view(T, H, P)
    out = torch.zeros(T, H, P)
    for i in range(len(slots)):
        t0, t1, s = int(cu_seq[i]), int(cu_seq[i + 1]), int(slots[i])
        if t1 <= t0:
            continue
        S = state[s].clone()
        for t in range(t0, t1):
            S = S * keep[t].unsqueeze(1) + vf[t].unsqueeze(2) * write[t].unsqueeze(1)
            out[t] = torch.einsum("hpn,hn->hp", S, qf[t])
        if write_state:
            state[s] = S
    out = _norm32(out, norm_w, eps, 0.0) * scale
    return out.reshape(T, H * P).to(q.dtype)


def xielu(z, ab):
    """a z^2 + z / 2 for z > 0, b (exp(z) - 1 - z) + z / 2 otherwise; ab = (a, b) float32."""
    n = z.clamp(max=0)
    return torch.where(z > 0, ab[0] * z * z, ab[1] * (torch.expm1(n) - n)) + 0.5 * z


def up_act(x, w, ab):
    return xielu(x.float() @ w.float().t(), ab).to(x.dtype)


def group_rms(x, w, groups: int, eps: float):
    """RMS norm in ``groups`` equal parts of a float32 row, times w."""
    v = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return (v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)).reshape(x.shape) * w


def resid_step(x, y, post_w, norm_w, groups: int, eps: float, dtype, conv=None):
    """x [T, H] float32 -> (x + norm(y), h): h = n + conv(n) with n the norm of the new x. y None: x as it is.
    ``conv`` = (taps [K, H] oldest first, history [slots, K - 1, H], cu_seq, slots, write_state) or None."""
    if y is not None:
        x = x + group_rms(y.float(), post_w, groups, eps)
    n = group_rms(x, norm_w, groups, eps)
    if conv is None:
        return x, n.to(dtype)
    taps, hist, cu, slots, write = conv
    K = taps.shape[0]
    h = torch.empty_like(n)
    for i in range(len(slots)):
        t0, t1 = int(cu[i]), int(cu[i + 1])
        if t1 <= t0:
            continue
        seq = torch.cat([hist[int(slots[i])], n[t0:t1]], 0)
        h[t0:t1] = n[t0:t1] + sum(taps[j] * seq[j:j + t1 - t0] for j in range(K))
        if write and K > 1:
            hist[int(slots[i])] = seq[seq.shape[0] - (K - 1):]
    return x, h.to(dtype)


def rotate_pairs(x, cos_sin, positions):
    """x [T, ..., D] float32: neighbouring columns (2i, 2i + 1) of the first cos_sin.shape[1] columns turn."""
    r = cos_sin.shape[1]
    cs = cos_sin[positions.long()].view(x.shape[0], *[1] * (x.dim() - 2), r)
    c, s = cs[..., :r // 2], cs[..., r // 2:]
    u, v = x[..., 0:r:2], x[..., 1:r:2]
    out = x.clone()
    out[..., 0:r:2], out[..., 1:r:2] = u * c - v * s, v * c + u * s
    return out


def latent_queries(q, kv, uk, norm_w, eps: float, cos_sin, positions, slots, cache, heads: int, dim: int, rot_dim: int):
    """Cache rows [norm(latent) | rotated key part] at the tokens' cells; returns [T, heads, rank + rot_dim]: queries in
    the latent space and their rotated part."""
    T, L = q.shape[0], norm_w.numel()
    kvf = kv.float()
    c = group_rms(kvf[:, :L], norm_w, 1, eps)
    row = torch.cat([c, rotate_pairs(kvf[:, L:L + rot_dim], cos_sin, positions)], 1).to(cache.dtype)
    valid = slots >= 0
    cache.view(-1, cache.shape[-1])[slots[valid], :L + rot_dim] = row[valid]
    qh = q.float().reshape(T, heads, dim + rot_dim)
    qa = torch.einsum("thd,hld->thl", qh[..., :dim], uk.float().view(heads, L, dim))
    return torch.cat([qa, rotate_pairs(qh[..., dim:], cos_sin, positions)], 2).to(q.dtype)


def latent_attention(q_abs, cache, block_table, ctx_lens, cu_q, scale: float, rank: int):
    """Causal attention of q_abs [T, heads, D] over cache rows [D, ...]; values are a row's first ``rank`` columns."""
    D = q_abs.shape[2]
    k = cache[..., :D]
    return paged_attention(q_abs, k, k, block_table, ctx_lens, cu_q, scale)[..., :rank]


def latent_values(o_lat, uv, gate):
    """Per-head value projection and output gate: gate [T, heads * vdim], [T, heads] or None."""
    T, H, L = o_lat.shape
    o = torch.einsum("thl,hvl->thv", o_lat.float(), uv.float().view(H, -1, L))
    if gate is not None:
        g = torch.sigmoid(gate.float())
        o = o * (g[:, :, None] if gate.shape[1] == H else g.view(o.shape))
    return o.reshape(T, -1).to(o_lat.dtype)


def head_linear(x, w, heads: int):
    """x in ``heads`` equal parts, each times its own matrix: w [heads * n, k]; float32 [T, heads * n]."""
    xh = x.float().view(x.shape[0], heads, -1)
    return torch.einsum("thk,hnk->thn", xh, w.float().view(heads, -1, xh.shape[2])).reshape(x.shape[0], -1)


def gated_recurrence(u, gates, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks: int, write_state: bool = True):
    """RG-LRU over the step's tokens: gates float32 [T, blocks, 2, width / blocks] (recurrence, input; before bias and
    sigmoid), a = exp(sigmoid(r) log_decay), S = a S + sqrt(1 - a^2) sigmoid(i) u; returns S * gelu(y + y_b)."""
    T, W = u.shape
    z = torch.sigmoid((gates.reshape(T, -1) + gates_b).view(T, blocks, 2, -1))
    r, i = z[:, :, 0].reshape(T, W), z[:, :, 1].reshape(T, W)
    la = r * log_decay
    a, b = torch.exp(la), torch.sqrt(-torch.expm1(2 * la)) * i * u.float()
    out = torch.empty(T, W, dtype=torch.float32, device=u.device)
    for n in range(len(slots)):
        S = state[int(slots[n])].clone()
        for t in range(int(cu_seq[n]), int(cu_seq[n + 1])):
            S = a[t] * S + b[t]
            out[t] = S
        if write_state:
            state[int(slots[n])] = S
    return (out * F.gelu(y.float() + y_b, approximate="tanh")).to(u.dtype)


def sample(logits, temperature, top_k, top_p, min_p, generator=None):
    """Host-order sampling for one row: temperature -> min-p -> top-k -> top-p -> draw."""
    lf = logits.float()
    if temperature <= 0:
        return int(torch.argmax(lf))
    p = torch.softmax(lf / temperature, dim=-1)
    if min_p and min_p > 0:
        p = torch.where(p >= min_p * p.max(), p, torch.zeros_like(p))
    if top_k and 0 < top_k < p.numel():
        kth = torch.topk(p, top_k).values[-1]
        p = torch.where(p >= kth, p, torch.zeros_like(p))
    if top_p is not None and top_p < 1.0:
        sp, si = torch.sort(p, descending=True)
        csum = torch.cumsum(sp, 0) / sp.sum()
        keep = (csum - sp / sp.sum()) < top_p
        mask = torch.zeros_like(p, dtype=torch.bool)
        mask[si[keep]] = True
        p = torch.where(mask, p, torch.zeros_like(p))
    p = p / p.sum()
    return int(torch.multinomial(p, 1, generator=generator))
