"""Ops: one function per kernel family.

CUDA tensors run the hand-written sm_100a kernels (``ops.sm100``; the extension is required, there is
no eager fallback on a GPU). CPU tensors run the float32 PyTorch reference (``ops.reference``), which
is both the test oracle and the back-end of the CPU engine used by the scheduler / cache / speculative
decoding tests.
"""
from __future__ import annotations

import torch

from . import reference as _ref
from . import sm100 as _sm

reference = _ref
sm100 = _sm


def _cuda(t) -> bool:
    return t.is_cuda


def linear(x, w, residual=None, out_dtype=None, out=None, tok_scale=None):
    """x @ w^T, each row times its ``tok_scale`` (float32 [T]), plus the residual."""
    if _cuda(x):
        return _sm.linear(x, w, residual=residual, out=out, out_dtype=out_dtype or getattr(x, "dtype", torch.bfloat16),
                          tok_scale=tok_scale)
    y = _ref.linear(x, w, residual=residual, out_dtype=out_dtype if tok_scale is None else torch.float32)
    if tok_scale is not None:
        y = (y * tok_scale[:, None]).to(out_dtype or x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def gate_up_act(x, w_gate_up, n_ff, act="silu", bias=None):
    """act(x Wg^T + bg) * (x Wu^T + bu); ``bias`` float32 [bg | bu], optional."""
    if bias is not None and _cuda(x):
        return _sm.gate_up_act(x, w_gate_up, n_ff, act=act, bias=bias)
    if _cuda(x):
        if act == "silu" or (act == "gelu_tanh" and isinstance(w_gate_up, torch.Tensor)):
            return _sm.gate_up_act(x, w_gate_up, n_ff, act=act)
        h = _sm.linear(x, w_gate_up)
        out = torch.empty(x.shape[0], n_ff, dtype=torch.bfloat16, device=x.device)
        _sm.ext().glu(h, out, n_ff, {"gelu_tanh": 1, "relu2": 2}[act])
        return out
    return _ref.gate_up_act(x, w_gate_up, n_ff, act, bias)


def rmsnorm(x, w, eps, w_offset=0.0, residual=None):
    """Returns (normed, summed)."""
    if _cuda(x):
        return _sm.rmsnorm(x, w, eps, w_offset, residual)
    return _ref.rmsnorm(x, w, eps, w_offset, residual)


def qk_norm_rope_append(qkv, n_q, n_kv, d, q_norm_w, k_norm_w, eps, w_offset, cos_sin, rot, positions, slots, k_cache,
                        v_cache, gated_q=False):
    """Returns (q [T, n_q, d], gate handle). On CUDA the gate stays inside ``qkv`` (handle = qkv)."""
    if _cuda(qkv):
        q = _sm.qk_norm_rope_append(qkv, n_q, n_kv, d, q_norm_w, k_norm_w, eps, w_offset, cos_sin, rot, positions,
                                    slots, k_cache, v_cache, gated_q)
        return q, (qkv if gated_q else None)
    return _ref.qk_norm_rope_append(qkv, n_q, n_kv, d, q_norm_w, k_norm_w, eps, w_offset, cos_sin, rot, positions,
                                    slots, k_cache, v_cache, gated_q)


def apply_output_gate(attn, gate, n_q, d):
    """attn [T, n_q, d] * sigmoid(gate)."""
    if _cuda(attn):
        return _sm.sigmoid_gate(attn, gate, n_q, d)
    return (attn.float() * torch.sigmoid(gate.float())).to(attn.dtype)


def paged_attention(q, k_cache, v_cache, block_table, ctx_lens, cu_q, max_q_len, scale, window=0, causal=True,
                    decode_splits=None, max_ctx=None, softcap=0.0, keep_first=0, sink=None, gate=None, out_scale=1.0, out=None):
    """Varlen paged attention; ``max_q_len == 1`` selects the flash-decoding kernel on CUDA. fp32 caches and head sizes
    the tensor-core kernels do not take run on the general kernel (causal only). ``softcap`` > 0: scores become
    softcap * tanh(score / softcap). ``keep_first``: first tokens that stay visible behind the window; ``sink`` [Hq]
    float32: exp(sink) joins the softmax's denominator; ``gate`` [T, Hq]: each head's output times its sigmoid; ``out_scale``
    multiplies the output; ``out`` [T, Hq * Dv] (rows may lie apart) takes it."""
    if keep_first or sink is not None or gate is not None or out is not None or out_scale != 1.0:
        if not causal or softcap:
            raise NotImplementedError("sinks, kept first tokens and output gates come with causal attention without a soft cap")
        if _cuda(q):
            return _sm.attention_ext(q, k_cache, v_cache, block_table, ctx_lens, cu_q, max_q_len, scale, window, keep_first,
                                     sink, gate, out_scale, out, decode_splits, max_ctx)
        o = _ref.paged_attention(q, k_cache, v_cache, block_table, ctx_lens, cu_q, scale, window, sinks=sink,
                                 keep_first=keep_first, gate=gate, out_scale=out_scale)
        if out is None:
            return o
        out.copy_(o.reshape(out.shape))
        return out
    if _cuda(q):
        if not _sm.attn_tc_ok(q, k_cache, v_cache):
            return _sm.paged_attn_general(q, k_cache, v_cache, block_table, ctx_lens, cu_q, scale, window, causal,
                                          softcap=softcap)
        if max_q_len == 1 and causal:
            return _sm.paged_decode(q, k_cache, v_cache, block_table, ctx_lens, scale, window, decode_splits, max_ctx,
                                    softcap=softcap)
        return _sm.prefill_attn(q, k_cache, v_cache, cu_q, ctx_lens, block_table, max_q_len, scale, window, causal,
                                softcap=softcap)
    return _ref.paged_attention(q, k_cache, v_cache, block_table, ctx_lens, cu_q, scale, window, causal, softcap=softcap)


def router_topk(logits, k, mode="softmax", renorm=True, route_scale=1.0, bias=None, n_group=1, topk_group=1):
    if _cuda(logits):
        return _sm.router_topk(logits, k, mode, renorm, route_scale, bias, n_group, topk_group)
    return _ref.router_topk(logits, k, mode, renorm, route_scale, bias, n_group, topk_group)


def router(x, w_router, k, mode="softmax", renorm=True, route_scale=1.0, bias=None, n_group=1, topk_group=1,
           e_lo=0, n_local=None, norm=None, group_top=2, gate_row=False, shared_slots=0, **gpu_kw):
    """Router projection + top-k. Returns an object that unpacks as ``ids, wts`` ([T, k] int32 / float32); on the
    GPU it may also carry the dense routing tables of a decode-sized step for the experts
    [e_lo, e_lo + n_local) of this rank (pass it on as ``routing=``). With ``norm=(weight, eps, w_offset)`` ``x`` is
    the raw residual stream: the RMSNorm runs first (inside the routing launch for decode-sized steps on the GPU)
    and the result's ``x_normed`` is the normalised input for the experts. ``gate_row``: the last row of ``w_router``
    gates the shared expert; the result's ``gate`` is its sigmoid [T] (None where the shared expert, stored as
    ``shared_slots`` experts behind the routed ones, rides in the dense routing tables)."""
    if _cuda(x):
        return _sm.router(x, w_router, k, mode, renorm, route_scale, bias, n_group, topk_group, norm, e_lo, n_local,
                          group_top=group_top, gate_row=gate_row, shared_slots=shared_slots, **gpu_kw)
    xn = None
    if norm is not None:
        xn, _ = _ref.rmsnorm(x, norm[0], norm[1], norm[2])
    logits = _ref.linear(x if xn is None else xn, w_router, out_dtype=torch.float32)
    gate = None
    if gate_row:
        logits, gate = logits[:, :-1], torch.sigmoid(logits[:, -1])
    ids, wts = _ref.router_topk(logits, k, mode, renorm, route_scale, bias, n_group, topk_group, group_top)
    r = _sm.Routing(ids, wts, None, xn)
    r.gate = gate
    return r


def _moe_experts_ungated(x, ids, wts, w_up, w_down, e_lo, shared, shared_gate, residual, norm, act="relu2", n_ff=None):
    """Experts the grouped kernels do not cover (un-gated squared ReLU, GELU-gated) on a GPU by tensor operations:
    pairs sorted by expert, one batched product per weight over padded per-expert groups."""
    T, H = x.shape
    E = w_up.shape[0]
    k = ids.shape[1]
    flat = ids.reshape(-1).long() - e_lo
    mine = (flat >= 0) & (flat < E)
    tok = torch.arange(T, device=x.device).repeat_interleave(k)
    key = torch.where(mine, flat, torch.full_like(flat, E))
    order = torch.argsort(key, stable=True)
    counts = torch.zeros(E + 1, dtype=torch.int64, device=x.device).scatter_add_(0, key, torch.ones_like(key))[:E]
    cap = T * k if T * k <= 64 else int(counts.max().item())          # small steps: no host read
    cap = max(cap, 1)
    starts = torch.cumsum(counts, 0) - counts
    pos = torch.arange(cap, device=x.device)[None, :]                 # [1, cap]
    src = (starts[:, None] + pos).clamp(max=T * k - 1)                # [E, cap] index into the sorted pairs
    live = pos < counts[:, None]
    pair = order[src]                                                 # [E, cap] pair index
    xg = x[tok[pair]] * live[..., None].to(x.dtype)                   # [E, cap, H]
    h = torch.bmm(xg, w_up.transpose(1, 2))
    if n_ff is not None and h.shape[-1] == 2 * n_ff:       # gated: [gate | up]
        h = (_ref.activation(h[..., :n_ff].float(), act) * h[..., n_ff:].float()).to(x.dtype)
    else:
        h = _ref.activation(h.float(), act).to(x.dtype)
    y = torch.bmm(h, w_down.transpose(1, 2)).float()                  # [E, cap, H]
    y = y * (wts.reshape(-1)[pair] * live).unsqueeze(-1)
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    out.index_add_(0, tok[pair].reshape(-1), y.reshape(-1, H))
    if shared is not None:
        s = shared.float()
        if shared_gate is not None:
            s = s * torch.sigmoid(shared_gate.float())[:, None]
        out = out + s
    if residual is not None:
        out = out + residual.float()
    out = out.to(x.dtype)
    if norm is None:
        return out
    return out, rmsnorm(out, norm[0], norm[1], norm[2])[0]


def moe_experts(x, ids, wts, w_gate_up, w_down, n_ff, act="silu", e_lo=0, shared=None, shared_gate=None,
                residual=None, out=None, norm=None, routing=None, defer_combine=False):
    """Routed experts (+ optional shared-expert output with sigmoid gate logits, + residual). Returns [T, H];
    with ``norm=(weight, eps, w_offset)`` returns (out, rmsnorm(out)): on the GPU the norm rides on the combine."""
    if _cuda(x) and isinstance(w_gate_up, torch.Tensor) and not _sm.tma_ok(x, w_gate_up, w_down):
        return _sm.moe_experts_plain(x, ids, wts, w_gate_up, w_down, n_ff, act, e_lo, shared, shared_gate, residual, norm,
                                     defer_combine)
    if _cuda(x) and act == "relu2" and defer_combine == "pairs" and isinstance(w_gate_up, torch.Tensor):
        return _sm.moe_experts(x, ids, wts, w_gate_up, w_down, n_ff, e_lo, None, shared, shared_gate, residual, out, norm,
                               routing if isinstance(routing, _sm.Routing) else None, defer_combine=defer_combine, act=act)
    if _cuda(x) and act != "silu":
        if act not in ("relu2", "gelu_tanh") or not isinstance(w_gate_up, torch.Tensor):
            raise NotImplementedError("the grouped expert kernels implement SwiGLU experts (squared-ReLU and GELU "
                                      "experts run through tensor operations)")
        # un-gated squared-ReLU experts (Nemotron-H) and GELU-gated experts (Gemma 4): no grouped kernel of their own
        # yet; the per-expert products run as tensor operations over the tokens of each expert, on the device,
        # without a host round trip per expert
        return _moe_experts_ungated(x, ids, wts, w_gate_up, w_down, e_lo, shared, shared_gate, residual, norm, act, n_ff)
    if _cuda(x):
        return _sm.moe_experts(x, ids, wts, w_gate_up, w_down, n_ff, e_lo, None, shared, shared_gate, residual, out,
                               norm, routing if isinstance(routing, _sm.Routing) else None,
                               defer_combine=defer_combine)
    y = _ref.moe_experts(x, ids, wts, w_gate_up, w_down, n_ff, act, e_lo, e_lo + w_gate_up.shape[0])
    if shared is not None:
        s = shared.float()
        if shared_gate is not None:
            s = s * torch.sigmoid(shared_gate.float())[:, None]
        y = y + s
    if residual is not None:
        y = y + residual.float()
    y = y.to(x.dtype)
    if norm is None:
        return y
    return y, _ref.rmsnorm(y, norm[0], norm[1], norm[2])[0]


def argmax(logits):
    if _cuda(logits):
        return _sm.argmax(logits)
    return _ref.argmax(logits)


def embed(ids, table):
    if _cuda(table) and table.dtype == torch.float32:
        return table.index_select(0, ids.long())
    if _cuda(table):
        return _sm.embed(ids.int(), table)
    return table[ids.long()]


def causal_conv1d_silu(x, w, bias, conv_state, cu_seq, slots, write_state=True, max_len=None, in_bias=None, silu=True):
    if _cuda(x):
        return _sm.causal_conv1d_silu(x, w, bias, conv_state, cu_seq, slots, write_state, max_len=max_len, in_bias=in_bias,
                                      silu=silu)
    return _ref.causal_conv1d_silu(x, w, bias, conv_state, cu_seq, slots, write_state, in_bias, silu)


def up_act(x, w, ab):
    """Un-gated feed-forward input: xIELU(x w^T) with the activation's two numbers ``ab`` (float32)."""
    return _sm.up_act(x, w, ab) if _cuda(x) else _ref.up_act(x, w, ab)


def up_relu2(x, w):
    """Un-gated feed-forward input: relu(x w^T)^2."""
    return _sm.linear(x, w, out_dtype=x.dtype, unary="relu2") if _cuda(x) else _ref.gate_up_act(x, w, w.shape[0], "relu2")


def prenorm_start(table, ids, pre_w, norm_w, eps, w_offset=0.0, raw=None):
    """Start of a pre-norm stack on one fp32 residual: x = embedding rows (``ids`` None: rows are given), normed with
    ``pre_w`` when given. Returns (x [T, H] float32, norm of x or None without ``norm_w``); ``raw`` takes x in the
    activation type."""
    if _cuda(table):
        return _sm.prenorm_step(None, (), 1.0, norm_w, eps, w_offset, raw, start=(table, ids, pre_w))
    x, h = _ref.prenorm_start(table if ids is None else table[ids.long()], pre_w, norm_w, eps, w_offset)
    if raw is not None:
        raw.copy_(x)
    return x, h


def prenorm_step(x, terms, mult, norm_w, eps, w_offset=0.0, raw=None, dtype=None):
    """Behind a sublayer: x + mult * (sum of its output ``terms`` [(tensor or ops.sm100.PendingCombine, scale)]) and the
    norm of that for the next one, in one launch; on CUDA ``x`` is updated in place. No terms: only the norm."""
    if _cuda(x):
        return _sm.prenorm_step(x, terms, mult, norm_w, eps, w_offset, raw, dtype=dtype)
    x, h = _ref.prenorm_step(x, terms, mult, norm_w, eps, w_offset, dtype)
    if raw is not None:
        raw.copy_(x)
    return x, h


def qkv_conv_append(proj, in_b, conv_w, conv_state, cu_seq, state_slots, q_norm, k_norm, norm_over, eps, rot, layout, positions,
                    slots, k_cache, v_cache, heads, write_state=True, max_len=None):
    """What lies between the q | k | v projection and the scores (see ``reference.qkv_conv_append``)."""
    args = (proj, in_b, conv_w, conv_state, cu_seq, state_slots, q_norm, k_norm, norm_over, eps, rot, layout, positions, slots,
            k_cache, v_cache, heads, write_state)
    return _sm.qkv_conv_append(*args, max_len=max_len) if _cuda(proj) else _ref.qkv_conv_append(*args)


def channel_delta(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H, G, dk, dv, write_state=True,
                  max_len=None, cu_host=None):
    """Gated delta rule with a decay per key channel (see ``reference.channel_delta``)."""
    args = (qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H, G, dk, dv, write_state)
    return _sm.channel_delta(*args, max_len=max_len, cu_host=cu_host) if _cuda(qkv) else _ref.channel_delta(*args)


def low_rank_pair(x, w, n0, rank):
    """x [T, 2 * rank] = a | g times w = [W_a (n0 rows); W_g]: (a W_a^T [T, n0], g W_g^T)."""
    if _cuda(x) and w.shape[0] == 2 * n0:
        y = torch.empty(x.shape[0] * 2, n0, dtype=x.dtype, device=x.device)
        _sm.head_linear(x, w, 2, n0, n0, rank, rank, y)
        y = y.view(x.shape[0], 2 * n0)
        return y[:, :n0], y[:, n0:]
    return linear(x[:, :rank], w[:n0]), linear(x[:, rank:], w[n0:])


def head_norm_gate(o, gate, w, eps, heads):
    """RMS norm of each head of o [T, heads * d], times w [d], times sigmoid(gate)."""
    if _cuda(o):
        return _sm.head_norm_gate(o, gate, w, eps, heads)
    return _ref.gated_rmsnorm(o.view(o.shape[0], heads, -1), gate.reshape(o.shape[0], heads, -1), w, eps,
                              "sigmoid").reshape(o.shape)


def depth_start(table, ids, layers: int, norm_w, eps, w_offset=0.0, average=True):
    """Start of a stack with parallel sublayers: x = embedding rows (``ids`` None: rows are given). Returns (x [T, H] float32,
    ops.sm100.DepthHistory with x as its first entry, or None without depth averages, norm of x)."""
    T = table.shape[0] if ids is None else ids.numel()
    hist = torch.empty(layers + 1 if average else 1, T, table.shape[1], dtype=torch.float32, device=table.device)
    if _cuda(table):
        _, h = _sm.prenorm_step(None, (), 1.0, norm_w, eps, w_offset, None, start=(table, ids, None), x_out=hist[0])
    else:
        x, h = _ref.prenorm_start(table if ids is None else table[ids.long()], None, norm_w, eps, w_offset)
        hist[0] = x
    return hist[0], _sm.DepthHistory(hist) if average else None, h


def depth_step(x, hist, i, y1, g1, b1, y2, g2, b2, y2_b, coefs, norm_w, eps, w_offset=0.0, rows=None):
    """Behind a layer with parallel sublayers (see ``reference.depth_step``), one launch; ``y2`` may be a
    ops.sm100.PendingCombine."""
    f = _sm.depth_step if _cuda(x) else _ref.depth_step
    return f(x, hist, i, y1, g1, b1, y2, g2, b2, y2_b, coefs, norm_w, eps, w_offset, rows)


def forget_scan(q, f, v, f_b, lower, state, cu_seq, slots, H, N, P, norm_w, eps, scale=1.0, write_state=True, max_len=None,
                cu_host=None, out=None):
    """HGRN2 state with the norm per head behind it (see ``reference.forget_scan``); ``out`` [T, H * P] may have rows that lie
    apart."""
    args = (q, f, v, f_b, lower, state, cu_seq, slots, H, N, P, norm_w, eps, scale, write_state)
    if _cuda(q):
        return _sm.forget_scan(*args, max_len=max_len, cu_host=cu_host, out=out)
    y = _ref.forget_scan(*args)
    return y if out is None else out.copy_(y)


def resid_start(table, ids, embed_scale, norm_w, groups, eps, conv=None, max_len=None):
    """Start of a stack with one fp32 residual: x = embedding rows * scale (``ids`` None: rows are given). Returns
    (x [T, H] float32, input of the first sublayer); ``conv`` as in ``reference.resid_step``."""
    if _cuda(table):
        return _sm.resid_step(None, None, None, norm_w, groups, eps, conv, start=(table, ids, embed_scale),
                              max_len=max_len)
    x = (table if ids is None else table[ids.long()]).float() * embed_scale
    return _ref.resid_step(x, None, None, norm_w, groups, eps, table.dtype, conv)


def resid_step(x, y, post_w, norm_w, groups, eps, conv=None, max_len=None):
    """Behind a sublayer with output y: x + norm(y), the norm of that and its input convolution, in one launch.
    Returns (new x, input of the next sublayer)."""
    if _cuda(x):
        return _sm.resid_step(x, y, post_w, norm_w, groups, eps, conv, max_len=max_len)
    return _ref.resid_step(x, y, post_w, norm_w, groups, eps, y.dtype, conv)


def latent_queries(q, kv, uk, norm_w, eps, cos_sin, positions, slots, cache, heads, dim, rot_dim):
    f = _sm.latent_queries if _cuda(q) else _ref.latent_queries
    return f(q, kv, uk, norm_w, eps, cos_sin, positions, slots, cache, heads, dim, rot_dim)


def latent_attention(q_abs, cache, block_table, ctx_lens, cu_q, max_q_len, scale, rank, rot_dim, max_ctx=None):
    if _cuda(q_abs):
        return _sm.latent_attention(q_abs, cache, block_table, ctx_lens, cu_q, max_q_len, scale, rank, rot_dim, max_ctx)
    return _ref.latent_attention(q_abs, cache, block_table, ctx_lens, cu_q, scale, rank)


def latent_values(o_lat, uv, gate):
    return _sm.latent_values(o_lat, uv, gate) if _cuda(o_lat) else _ref.latent_values(o_lat, uv, gate)


def block_gates(u, w, blocks):
    """Block-diagonal product, float32 result [T, rows of w]."""
    return _sm.block_gates(u, w, blocks) if _cuda(u) else _ref.head_linear(u, w, blocks)


def gated_recurrence(u, gates, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks, write_state=True, max_len=None,
                     cu_host=None):
    if _cuda(u):
        return _sm.gated_recurrence(u, gates, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks, write_state,
                                    max_len, cu_host)
    return _ref.gated_recurrence(u, gates, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks, write_state)


def hyper_start(table, ids, streams, in_w, norm_w, eps, w_offset=0.0):
    """Hyper-connections with static weights: the streams start as the embedding rows (``ids`` None: the rows are given
    in ``table``). Returns (streams [T, S, H] float32, normed input of the first sublayer)."""
    if _cuda(table):
        return _sm.hyper_start(table, ids, streams, in_w, norm_w, eps, w_offset)
    return _ref.hyper_start(table if ids is None else table[ids.long()], streams, in_w, norm_w, eps, w_offset)


def hyper_step(X, terms, mix, out_w, in_w, norm_w, eps, w_offset=0.0):
    """Stream update behind a sublayer, input mix and norm of the next one, in one launch; on CUDA ``X`` is updated in
    place. ``terms``: [(sublayer output, scale)], at most two; an ``ops.sm100.PendingCombine`` counts as one."""
    if _cuda(X):
        return _sm.hyper_step(X, terms, mix, out_w, in_w, norm_w, eps, w_offset)
    return _ref.hyper_step(X, terms, mix, out_w, in_w, norm_w, eps, w_offset)


def qkv_norm_append(q, k, v, q_norm, k_norm, eps, slots, k_cache, v_cache):
    if _cuda(q):
        return _sm.qkv_norm_append(q, k, v, q_norm, k_norm, eps, slots, k_cache, v_cache)
    return _ref.qkv_norm_append(q, k, v, q_norm, k_norm, eps, slots, k_cache, v_cache)


def linear_scan(q, k, v, state, cu_seq, slots, H, G, N, P, max_len=None, cu_host=None, **kw):
    """Decayed linear-attention state (see ``reference.linear_scan``)."""
    if _cuda(q):
        return _sm.linear_scan(q, k, v, state, cu_seq, slots, H, G, N, P, max_len=max_len, cu_host=cu_host, **kw)
    return _ref.linear_scan(q, k, v, state, cu_seq, slots, H, G, N, P, **kw)


def group_norm_gate(y, gate, w, eps, groups=1):
    if _cuda(y):
        return _sm.group_norm_gate(y, gate, w, eps, groups)
    return _ref.group_norm_gate(y, gate, w, eps, groups)


def gdn_gates(a, b, A, dt_bias):
    if _cuda(a):
        return _sm.gdn_gates(a, b, A, dt_bias)
    return _ref.gdn_gates(a, b, A, dt_bias)


def gdn_recurrent(qkv, g, beta, state, cu_seq, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps=1e-6,
                  write_state=True, cu_host=None):
    if _cuda(qkv):
        return _sm.gdn_recurrent(qkv, g, beta, state, cu_seq, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps,
                                 write_state, cu_host=cu_host)
    return _ref.gdn_recurrent(qkv, g, beta, state, cu_seq, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps,
                              write_state)


def gated_rmsnorm(o, z, w, eps, act="silu"):
    if _cuda(o):
        return _sm.gated_rmsnorm(o, z, w, eps, act)
    return _ref.gated_rmsnorm(o, z.reshape(o.shape), w, eps, act)
