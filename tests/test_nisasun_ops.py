"""Each mechanism of the Nisasun design alone, against the functions of ``nisasun_oracle`` (float64): on CPU the
reference ops, on a GPU the kernels in fp32 and bf16."""
import pytest
import torch

import nisasun_case as nc
import nisasun_oracle as oracle
from legion_b200 import ops

gpu = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda:0", torch.float32, id="gpu-f32", marks=gpu),
         pytest.param("cuda:0", torch.bfloat16, id="gpu-bf16", marks=gpu)]
BF16 = [WHERE[2]]


def rnd(*shape, seed=0, dtype=torch.float32, device="cpu", k=1.0):
    """Random values that are exact in ``dtype``, so that only the op under test rounds."""
    t = torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * k
    return t.to(dtype).to(device)


def d(t):
    return t.detach().cpu().double()


def close(got, want, dtype, tol32=2e-5, tol16=1e-2):
    scale = want.abs().max().clamp_min(1e-6)
    e = float((d(got) - want).abs().max() / scale)
    assert e < (tol32 if dtype == torch.float32 else tol16), e


def status_ok(device):
    if device != "cpu":
        torch.cuda.synchronize()
        assert ops.sm100.Workspace.get(device).check() == 0


# ------------------------------------------------------------------------------------------- hyper-connections
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("S,H,T", [(1, 64, 5), (2, 100, 3), (3, 256, 7), (4, 2048, 33), (5, 36, 1), (8, 129, 4), (11, 24, 6)])
def test_hyper_connections(device, dtype, S, H, T):
    eps = 1e-5
    emb = rnd(20, H, seed=1, dtype=dtype, device=device)
    ids = torch.randint(0, 20, (T,), generator=torch.Generator().manual_seed(2)).int().to(device)
    inw, outw, mix = (rnd(*s, seed=3 + i, device=device) for i, s in enumerate([(S,), (S,), (S, S)]))
    in2, n1, n2 = rnd(S, seed=6, device=device), rnd(H, seed=7, k=0.2, device=device), rnd(H, seed=8, k=0.2, device=device)
    y0, y1 = rnd(T, H, seed=9, dtype=dtype, device=device), rnd(T, H, seed=10, dtype=dtype, device=device)
    X, h = ops.hyper_start(emb, ids, S, inw, n1, eps, 1.0)
    X0 = torch.stack([d(emb)[ids.cpu().long()]] * S, 1)
    assert torch.equal(d(X), X0)
    close(h, oracle.stream_norm(torch.einsum("s,tsd->td", d(inw), X0), d(n1), eps), dtype)
    Xs = rnd(T, S, H, seed=11, device=device)
    w = {"c.in": d(inw), "c.out": d(outw), "c.mix": d(mix)}
    seen = []
    want = oracle.hyper(d(Xs), w, "c", d(n1), lambda u: seen.append(u) or (0.7 * d(y0) - 1.3 * d(y1)), eps)
    Xn, h = ops.hyper_step(Xs.clone(), [(y0, 0.7), (y1, -1.3)], mix, outw, in2, n2, eps, 1.0)
    close(Xn, want, torch.float32, 2e-6)
    close(h, oracle.stream_norm(torch.einsum("s,tsd->td", d(in2), want), d(n2), eps), dtype)
    _, h = ops.hyper_step(Xs.clone(), [(y0, 0.7), (y1, -1.3)], mix, outw, None, n2, eps, 1.0)     # the last one
    close(h, oracle.stream_norm(want.sum(1), d(n2), eps), dtype)


# ------------------------------------------------------------------------------------------- windowed attention
def paged(k, v, page, device, dtype):
    """Keys and values of sequences in shuffled pages of a pool full of large values: a cell that must not be read
    shows."""
    n_pages = [-(-x.shape[0] // page) for x in k]
    total = sum(n_pages) + 3
    order = torch.randperm(total, generator=torch.Generator().manual_seed(5)).tolist()
    kc = torch.full((total, page, k[0].shape[1], k[0].shape[2]), 30.0, device=device, dtype=dtype)
    vc = torch.full((total, page, v[0].shape[1], v[0].shape[2]), 1e4, device=device, dtype=dtype)
    bt = torch.zeros(len(k), max(n_pages), dtype=torch.int32)
    for i, n in enumerate(n_pages):
        for j in range(n):
            b = order.pop()
            bt[i, j] = b
            m = min(page, k[i].shape[0] - j * page)
            kc[b, :m], vc[b, :m] = k[i][j * page:j * page + m].to(device), v[i][j * page:j * page + m].to(device)
    return kc, vc, bt.to(device)


def windowed(q, k, v, scale, window):
    """q [T, H, dk] = the last rows of the keys' sequence."""
    T, H = q.shape[:2]
    n, G = k.shape[0], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float64)
    for t in range(T):
        i = n - T + t
        lo = max(0, i - window + 1)
        for h in range(H):
            s = k[lo:i + 1, h // (H // G)] @ q[t, h] * scale
            e = torch.exp(s - s.max())
            out[t, h] = (e / e.sum()) @ v[lo:i + 1, h // (H // G)]
    return out


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 88, 128), (6, 3, 40, 72), (2, 2, 64, 256), (3, 1, 136, 24), (2, 1, 13, 19),
                                       (16, 1, 128, 128), (4, 4, 256, 64), (4, 2, 120, 192), (2, 1, 40, 136),
                                       (2, 2, 168, 184)])
def test_windowed_attention_prompts_and_decode(device, dtype, H, G, dk, dv):
    lens, qlens = [200, 64, 1, 131], [70, 64, 1, 2]
    k = [rnd(n, G, dk, seed=i, dtype=dtype) for i, n in enumerate(lens)]
    v = [rnd(n, G, dv, seed=20 + i, dtype=dtype) for i, n in enumerate(lens)]
    kc, vc, bt = paged(k, v, 64, device, dtype)
    ctx = torch.tensor(lens, dtype=torch.int32, device=device)
    for ql in (qlens, [1] * 4):
        q = [rnd(n, H, dk, seed=40 + i, dtype=dtype) for i, n in enumerate(ql)]
        cu = torch.tensor([0] + torch.tensor(ql).cumsum(0).tolist(), dtype=torch.int32, device=device)
        for window in (1, 2, 63, 64, 65, 100, 1000):
            got = ops.paged_attention(torch.cat(q).to(device), kc, vc, bt, ctx, cu, max(ql), 0.31 * dk ** -0.5, window=window,
                                      max_ctx=200)
            want = torch.cat([windowed(d(a), d(b), d(c), 0.31 * dk ** -0.5, window) for a, b, c in zip(q, k, v)])
            close(got, want, dtype)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("dk,dv", [(112, 160), (20, 12)])
@pytest.mark.parametrize("window", [1, 8, 64, 65, 127, 128, 129, 300])
def test_one_key_at_the_window_edge(device, dtype, dk, dv, window):
    """One key scores far above all others and its value is marked: it decides the output exactly as long as it is
    inside the window, wherever pages end, in prompts and in decoding."""
    n = 420
    for at in (0, 63, 64, 100):
        k = rnd(n, 1, dk, seed=1, dtype=dtype, k=0.05)
        v = rnd(n, 1, dv, seed=2, dtype=dtype, k=0.1)
        k[at, 0], v[at, 0] = 4.0, 50.0
        kc, vc, bt = paged([k], [v], 64, device, dtype)
        last = at + window - 1                       # the last position that sees it
        for i in (last, last + 1):
            if i >= n:
                continue
            ctx = torch.tensor([i + 1], dtype=torch.int32, device=device)
            for ql in {1, min(2, i + 1), min(90, i + 1)}:
                q = torch.full((ql, 1, dk), 4.0, dtype=dtype, device=device)
                cu = torch.tensor([0, ql], dtype=torch.int32, device=device)
                o = ops.paged_attention(q, kc, vc, bt, ctx, cu, ql, 1.0, window=window, max_ctx=n)
                sees = d(o)[-1].mean() > 40
                assert sees == (i == last), (at, i, ql)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_head_norms_and_append(device, dtype):
    H, G, dk, dv, T = 6, 2, 40, 24, 9
    proj = rnd(T, H * dk + G * (dk + dv) + 8, seed=1, dtype=dtype, device=device)
    qw, kw = 1 + rnd(dk, seed=2, device=device, k=0.3), 1 + rnd(dk, seed=3, device=device, k=0.3)
    kc, vc = torch.zeros(2, 64, G, dk, dtype=dtype, device=device), torch.zeros(2, 64, G, dv, dtype=dtype, device=device)
    slots = torch.tensor([63, 64, 0, 127, -1, 5, 7, 9, 100], device=device)
    a, b, c = H * dk, (H + G) * dk, (H + G) * dk + G * dv
    q = ops.qkv_norm_append(proj[:, :a], proj[:, a:b], proj[:, b:c], qw, kw, 1e-5, slots, kc, vc)
    close(q, oracle.rms(d(proj[:, :a]).view(T, H, dk), 1e-5) * d(qw), dtype)
    keep = [i for i in range(T) if i != 4]
    cells = slots[keep]
    close(kc.view(-1, G, dk)[cells], (oracle.rms(d(proj[:, a:b]).view(T, G, dk), 1e-5) * d(kw))[keep], dtype)
    assert torch.equal(d(vc.view(-1, G, dv)[cells]), d(proj[:, b:c]).view(T, G, dv)[keep])
    assert float(vc.float().abs().sum()) == pytest.approx(float(proj[:, b:c][keep].float().abs().sum()), rel=1e-5)


# ------------------------------------------------------------------------------------------- recurrent state
def scan_case(H, G, N, P, lens, seed, device, dtype, kind):
    T = sum(lens)
    slots = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(seed))[:len(lens)].int().to(device)
    state = rnd(len(lens) + 2, H, P, N, seed=seed + 1, device=device)
    cu = [0] + torch.tensor(lens).cumsum(0).tolist()
    pad = rnd(T, 2 * G * N + H * P + 8, seed=seed + 2, dtype=dtype, device=device, k=0.7)
    q, k, v = pad[:, :G * N], pad[:, G * N:2 * G * N], pad[:, 2 * G * N:2 * G * N + H * P]
    kw = {}
    if kind == "constant":
        kw = dict(decay=torch.tensor([1 - 0.6 ** (1 + 2 * h) for h in range(H)], device=device), silu_in=True)
    else:
        kw = dict(dt=rnd(T, H, seed=seed + 3, dtype=dtype, device=device), dt_bias=rnd(H, seed=seed + 4, device=device),
                  A=-torch.exp(rnd(H, seed=seed + 5)).to(device), D=rnd(H, seed=seed + 6, device=device),
                  z=rnd(T, H * P, seed=seed + 7, dtype=dtype, device=device))
    return q, k, v, state, torch.tensor(cu, dtype=torch.int32, device=device), slots, cu, kw


def scan_expected(q, k, v, state, cu, slots, H, G, N, P, kw):
    T = q.shape[0]
    q, k, v = d(q).view(T, G, N), d(k).view(T, G, N), d(v).view(T, H, P)
    if kw.get("silu_in"):
        q, k, v = oracle.silu(q), oracle.silu(k), oracle.silu(v)
    grp = [h // (H // G) for h in range(H)]
    vs = v
    if "decay" in kw:
        dec = d(kw["decay"]).expand(T, H)
    else:
        a = d(kw["dt"]) + d(kw["dt_bias"])
        dt = torch.clamp(a, min=0) + torch.log1p(torch.exp(-a.abs()))
        dec, vs = torch.exp(dt * d(kw["A"])), v * dt[..., None]
    out, states = torch.zeros(T, H, P, dtype=torch.float64), d(state)
    for i, s in enumerate(slots.tolist()):
        t0, t1 = cu[i], cu[i + 1]
        o, S = oracle.decayed_outer_products(q[t0:t1, grp], k[t0:t1, grp], vs[t0:t1], dec[t0:t1], states[s].transpose(1, 2))
        out[t0:t1] = o
        states[s] = S.transpose(1, 2)
    if "D" in kw:
        out = out + d(kw["D"])[:, None] * v
    out = out.reshape(T, H * P)
    if "z" in kw:
        out = out * oracle.silu(d(kw["z"]))
    return out, states


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("kind", ["constant", "selective"])
@pytest.mark.parametrize("H,G,N,P", [(6, 2, 32, 40), (3, 3, 48, 64), (2, 1, 13, 19), (2, 2, 128, 128), (4, 1, 40, 160)])
def test_linear_state(device, dtype, kind, H, G, N, P):
    if kind == "constant":
        G = H
    lens = [5, 1, 2, 40]
    q, k, v, state, cu, slots, cu_h, kw = scan_case(H, G, N, P, lens, 3, device, dtype, kind)
    want, states = scan_expected(q, k, v, state, cu_h, slots, H, G, N, P, kw)
    frozen = state.clone()
    ops.linear_scan(q, k, v, frozen, cu, slots, H, G, N, P, max_len=40, cu_host=cu_h, write_state=False, **kw)
    assert torch.equal(frozen, state)
    got = ops.linear_scan(q, k, v, state, cu, slots, H, G, N, P, max_len=40, cu_host=cu_h, **kw)
    close(got, want, dtype)
    close(state, states, torch.float32)             # the state stays fp32 whatever the activations are


@pytest.mark.parametrize("device,dtype", BF16)
@pytest.mark.parametrize("kind", ["constant", "selective"])
@pytest.mark.parametrize("H,G,N,P", [(6, 2, 32, 40), (3, 3, 48, 64), (2, 1, 13, 19), (2, 2, 128, 128), (4, 1, 40, 160),
                                     (2, 1, 100, 90)])
def test_linear_state_in_chunks(device, dtype, kind, H, G, N, P):
    """The tensor-core form: whole chunks, chunk edges, single tokens beside them, carried states; the state keeps far
    more than bf16 accuracy."""
    if kind == "constant":
        G = H
    lens = [300, 1, 128, 129, 2, 127, 64, 8, 9]
    q, k, v, state, cu, slots, cu_h, kw = scan_case(H, G, N, P, lens, 8, device, dtype, kind)
    want, states = scan_expected(q, k, v, state, cu_h, slots, H, G, N, P, kw)
    got = ops.sm100.linear_scan(q, k, v, state, cu, slots, H, G, N, P, cu_host=cu_h, chunked=True, **kw)
    status_ok(device)
    close(got, want, dtype)
    if kind == "selective":                         # operands exact in bf16: only the split operands round
        close(state, states, torch.float32, 1e-4)
    else:                                           # silu(k) and silu(v) are rounded to bf16 in front of the product
        close(state, states, dtype, tol16=6e-3)


@pytest.mark.parametrize("device,dtype", WHERE[1:])
@pytest.mark.parametrize("H,G,N,P,K", [(6, 2, 32, 40, 4), (6, 3, 16, 24, 1), (4, 4, 128, 64, 2), (8, 1, 40, 130, 9)])
def test_ssd_decode_step(device, dtype, H, G, N, P, K):
    """The fused decode launch against convolution and scan one after the other, several steps in a row."""
    n, C = 5, H * P + 2 * G * N
    slots = torch.tensor([3, 0, 6, 1, 4], dtype=torch.int32, device=device)
    cu = torch.arange(n + 1, dtype=torch.int32, device=device)
    cw, cb = rnd(C, K, seed=1, device=device, k=0.5), rnd(C, seed=2, device=device)
    dtb, A, D = rnd(H, seed=3, device=device), -torch.exp(rnd(H, seed=4)).to(device), rnd(H, seed=5, device=device)
    conv = rnd(7, C, K - 1, seed=6, device=device)
    state = rnd(7, H, P, N, seed=7, device=device)
    conv2, state2 = conv.cpu().clone(), state.cpu().clone()
    for step in range(3):
        proj = rnd(n, H * P + C + H, seed=30 + step, dtype=dtype, device=device)
        z, xbc, dt = proj[:, :H * P], proj[:, H * P:H * P + C], proj[:, H * P + C:]
        got = ops.sm100.ssd_decode(xbc, cw, cb, conv, dt, dtb, A, D, z, state, cu, slots, H, G, N, P)
        p = proj.cpu().float()
        z2, xbc2, dt2 = p[:, :H * P], p[:, H * P:H * P + C], p[:, H * P + C:]
        c = ops.reference.causal_conv1d_silu(xbc2, cw.cpu(), cb.cpu(), conv2, cu.cpu(), slots.cpu())
        want = ops.reference.linear_scan(c[:, H * P + G * N:], c[:, H * P:H * P + G * N], c[:, :H * P], state2, cu.cpu(),
                                         slots.cpu(), H, G, N, P, dt=dt2, dt_bias=dtb.cpu(), A=A.cpu(), D=D.cpu(), z=z2)
        close(got, want.double(), dtype)
        close(state, state2.double(), torch.float32)
        assert torch.allclose(conv.cpu(), conv2)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("K", [1, 2, 4, 5, 9])
def test_short_convolution_in_portions(device, dtype, K):
    C, T = 50, 170
    x = rnd(T, C, seed=1, dtype=dtype, device=device)
    w, b = rnd(C, K, seed=2, device=device, k=0.5), rnd(C, seed=3, device=device)
    want = oracle.silu(oracle.short_conv(d(x), d(w), d(b)))
    for cuts in ([170], [1] * 6 + [164], [2, 3, 1, 100, 64], [90, 2, 78]):
        hist = torch.zeros(3, C, K - 1, device=device)
        slot = torch.tensor([2], dtype=torch.int32, device=device)
        out, t = [], 0
        for c in cuts:
            cu = torch.tensor([0, c], dtype=torch.int32, device=device)
            out.append(ops.causal_conv1d_silu(x[t:t + c], w, b, hist, cu, slot, max_len=c))
            t += c
        close(torch.cat(out), want, dtype)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("C,groups", [(96, 1), (96, 4), (90, 5), (2048, 8)])
def test_group_norm_and_gate(device, dtype, C, groups):
    y, g = rnd(7, C, seed=1, dtype=dtype, device=device), rnd(7, C + 8, seed=2, dtype=dtype, device=device)[:, :C]
    w = 1 + rnd(C, seed=3, device=device, k=0.3)
    n = oracle.rms(d(y).view(7, groups, -1), 1e-5).reshape(7, C) * d(w)
    close(ops.group_norm_gate(y, None, w, 1e-5, groups), n, dtype)
    close(ops.group_norm_gate(y, g, w, 1e-5, groups), n / (1 + torch.exp(-d(g))), dtype)


# ------------------------------------------------------------------------------------------- feed-forward parts
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T", [3, 64, 65, 200])
@pytest.mark.parametrize("E,top,count,keep", [(15, 4, 5, 3), (8, 2, 2, 1), (5, 1, 1, 1), (64, 6, 8, 3), (6, 3, 6, 4)])
def test_router_groups_and_correction(device, dtype, T, E, top, count, keep):
    W = 64
    h = rnd(T, W, seed=1, dtype=dtype, device=device)
    wr = rnd(E, W, seed=2, dtype=dtype, device=device, k=0.5)
    corr = (rnd(E, seed=3, k=0.4) - 0.4).to(device)            # selection scores of either sign
    z = d(h) @ d(wr).T
    s = torch.softmax(z, -1)
    spec = {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}
    ids, wts = ops.router(h, wr, top, "softmax_bias", False, 1.0, corr, count, keep, group_top=1)
    assert bool((s + d(corr) < 0).any())
    for t in range(T):
        want = oracle.route(s[t], d(corr), spec)
        got = ids[t].tolist()
        if set(got) != set(want):                              # only where two selection scores nearly tie
            assert device != "cpu" and t < T and dtype == torch.bfloat16, (t, got, want)
            continue
        for e, x in zip(got, wts[t].tolist()):
            assert x == pytest.approx(float(s[t, e]), rel=2e-3, abs=1e-6)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T", [5, 90])
@pytest.mark.parametrize("W,ff,E", [(96, 40, 6), (50, 27, 3), (256, 128, 8)])
def test_experts_and_dense(device, dtype, T, W, ff, E):
    cfg = nc.config(W, 11, 1, [nc.lightning(1, 8, 8, nc.moe(E, 2, ff))])
    w = nc.make_weights(cfg, 4)
    spec = cfg["layers"][0]["mlp"]
    h = rnd(T, W, seed=1, dtype=torch.bfloat16).to(dtype)
    want = oracle.moe_ffn(d(h), {k: d(v) for k, v in w.items()}, "l0.mlp", spec)
    to = lambda t: t.to(dtype).to(device)                     # noqa: E731
    gu = to(torch.stack([torch.cat([w[f"l0.mlp.e{e}.gate"], w[f"l0.mlp.e{e}.up"]]) for e in range(E)]))
    dn = to(torch.stack([w[f"l0.mlp.e{e}.down"] for e in range(E)]))
    x = h.to(device)
    r = ops.router(x, to(w["l0.mlp.router"]), 2, "softmax_bias", False, 1.0, w["l0.mlp.correction"].float().to(device), 1, 1,
                   group_top=1)
    y = ops.moe_experts(x, r.ids, r.wts, gu, dn, ff, "silu", routing=r, defer_combine="pairs")
    X = torch.zeros(T, 1, W, device=device)
    one, zero = torch.ones(1, device=device), torch.zeros(W, device=device)
    X, _ = ops.hyper_step(X, [(y, 1.0)], torch.zeros(1, 1, device=device), one, one, zero, 1e-5, 1.0)
    close(X[:, 0], want, dtype, tol16=2e-2)
    g, u, dw = w["l0.mlp.e0.gate"], w["l0.mlp.e0.up"], w["l0.mlp.e0.down"]
    got = ops.linear(ops.gate_up_act(x, to(torch.cat([g, u])), ff, "gelu_tanh"), to(dw))
    close(got, oracle.dense_ffn(d(h), {"p.gate": d(g), "p.up": d(u), "p.down": d(dw)}, "p"), dtype)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,K,N", [(1, 90, 33), (40, 64, 100), (33, 13, 7), (130, 300, 65)])
def test_matrix_products_of_any_size(device, dtype, T, K, N):
    x, w = rnd(T, K, seed=1, dtype=dtype, device=device), rnd(N, K, seed=2, dtype=dtype, device=device)
    res = rnd(T, N, seed=3, dtype=dtype, device=device)
    close(ops.linear(x, w, out_dtype=torch.float32), d(x) @ d(w).T, torch.float32)
    close(ops.linear(x, w, residual=res), d(x) @ d(w).T + d(res), dtype)
