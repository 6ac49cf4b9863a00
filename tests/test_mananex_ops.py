"""Each mechanism of the Mananex design alone, against the functions of ``mananex_oracle`` (float64): on CPU the reference
ops, on a GPU the kernels in fp32 and bf16."""
import math

import pytest
import torch

import mananex_oracle as oracle
from legion_b200 import ops
from legion_b200.config import DenseSpec, LayerSpec, ModelConfig, MoeSpec, RotarySpec, SsdSpec

gpu = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda:0", torch.float32, id="gpu-f32", marks=gpu),
         pytest.param("cuda:0", torch.bfloat16, id="gpu-bf16", marks=gpu)]


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


def i32(x, device):
    return torch.tensor(x, dtype=torch.int32, device=device)


def portions(lens, cuts):
    """Steps of [(sequence, first token, tokens)] that feed every sequence in its own cuts."""
    at, steps, n = [0] * len(lens), [], 0
    while any(a < m for a, m in zip(at, lens)):
        step = []
        for i, m in enumerate(lens):
            c = min(cuts[i][n % len(cuts[i])], m - at[i])
            if c > 0:
                step.append((i, at[i], c))
                at[i] += c
        steps.append(step)
        n += 1
    return steps


def bounds(step, device):
    return i32([0] + torch.tensor([c for _, _, c in step]).cumsum(0).tolist(), device)


# ------------------------------------------------------------------------------------------- rotation, cache append
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,G,dk,dv,dims,base", [(6, 2, 40, 24, 24, 1e4), (1, 1, 21, 11, 10, 50.0), (16, 4, 128, 128, 64, 1e6),
                                                 (3, 1, 17, 35, 2, 1e3), (4, 4, 32, 48, 32, 100.0), (2, 1, 16, 8, 0, 1.0)])
@pytest.mark.parametrize("lens", [[1, 1, 1], [5, 1, 33], [64]])
def test_rotated_rows_on_their_way_to_the_cache(device, dtype, H, G, dk, dv, dims, base, lens):
    """Neighbouring columns of q and k turn, the rest and v pass unchanged, k and v land in their cells (a negative one drops
    them)."""
    T, ld = sum(lens), (H + G) * dk + G * dv + 16
    proj = rnd(T, ld, seed=1, dtype=dtype)
    pos = [p for i, n in enumerate(lens) for p in range(7 * i + 3, 7 * i + 3 + n)]
    C = (H + G) * dk + G * dv
    q = d(proj)[:, :H * dk].view(T, H, dk)
    k, v = d(proj)[:, H * dk:(H + G) * dk].view(T, G, dk), d(proj)[:, (H + G) * dk:C].view(T, G, dv)
    rot, table, want_q, want_k = {"dims": dims, "base": base}, None, q, k
    if dims:
        want_q, want_k = oracle.rotate(q, pos, rot), oracle.rotate(k, pos, rot)
        table = ops.reference.rope_cos_sin(128, dims, base, None).to(device)
    perm = torch.randperm(3 * 64, generator=torch.Generator().manual_seed(2))[:T]
    cells = perm.clone()
    cells[T // 2] = -1 if T > 1 else cells[T // 2]
    kc, vc = rnd(3, 64, G, dk, seed=3, dtype=dtype), rnd(3, 64, G, dv, seed=4, dtype=dtype)
    k_dev, v_dev = kc.to(device), vc.to(device)
    slots = i32(list(range(len(lens))), device)
    got = ops.qkv_conv_append(proj.to(device)[:, :C], None, None, None, i32([0] + torch.tensor(lens).cumsum(0).tolist(), device),
                              slots, None, None, "head", 1e-5, table, "pairs", i32(pos, device), cells.to(device), k_dev, v_dev, H,
                              max_len=max(lens))
    close(got, want_q, dtype)
    want_kc, want_vc = d(kc).view(-1, G, dk), d(vc).view(-1, G, dv)
    ok = cells >= 0
    want_kc[cells[ok]], want_vc[cells[ok]] = want_k[ok], v[ok]
    close(k_dev.view(-1, G, dk), want_kc, dtype)
    assert torch.equal(d(v_dev).view(-1, G, dv), want_vc)


@pytest.mark.parametrize("dims,base", [(2, 10.0), (16, 2e5), (24, 1e4), (128, 1e6)])
def test_rotation_frequencies(dims, base):
    from legion_b200.models.decoder import Decoder
    dec = Decoder.__new__(Decoder)
    dec._rot, dec.device = {}, torch.device("cpu")
    table = dec.rotary_table(RotarySpec(dims, base), 500)
    x = torch.zeros(500, 1, dims, dtype=torch.float64)
    x[:, :, 0::2] = 1.0                                        # (1, 0) turns into (cos, sin)
    y = oracle.rotate(x, range(500), {"dims": dims, "base": base})[:, 0]
    assert float((table.double() - torch.cat([y[:, 0::2], y[:, 1::2]], 1)).abs().max()) < 1e-6


# ------------------------------------------------------------------------------------------- attention
def paged(keys, vals, page, dtype, device, seed=9):
    """Sequences' keys and values [T, G, d] in shuffled pages; unused cells hold large values."""
    need = [-(-k.shape[0] // page) for k in keys]
    order = torch.randperm(sum(need) + 2, generator=torch.Generator().manual_seed(seed)).tolist()
    G, dk, dv = keys[0].shape[1], keys[0].shape[2], vals[0].shape[2]
    kc = torch.full((sum(need) + 2, page, G, dk), 30.0, dtype=dtype)
    vc = torch.full((sum(need) + 2, page, G, dv), 30.0, dtype=dtype)
    table = torch.zeros(len(keys), max(need), dtype=torch.int32)
    for i, (k, v) in enumerate(zip(keys, vals)):
        for b in range(need[i]):
            p = order.pop()
            table[i, b] = p
            n = min(page, k.shape[0] - b * page)
            kc[p, :n], vc[p, :n] = k[b * page:b * page + n].to(dtype), v[b * page:b * page + n].to(dtype)
    return kc.to(device), vc.to(device), table.to(device)


SHAPES = [(6, 2, 40, 24), (1, 1, 21, 11), (16, 4, 128, 128), (8, 8, 64, 64), (4, 2, 96, 200), (2, 1, 200, 72), (17, 1, 64, 40)]


def run_attention(device, dtype, H, G, dk, dv, lens, ctx, window, keep, scale=0.3, sink_at=0.5, out_scale=0.7, spike=None, gated=True):
    """Queries are the last ``lens`` tokens of sequences of ``ctx`` tokens; ``spike`` (sequence, key): one key that stands out
    for every query. Returns (got, expected) per sequence."""
    page, T = 64, sum(lens)
    keys = [rnd(c, G, dk, seed=10 + i, dtype=dtype) for i, c in enumerate(ctx)]
    vals = [rnd(c, G, dv, seed=30 + i, dtype=dtype) for i, c in enumerate(ctx)]
    q = rnd(T, H, dk, seed=50, dtype=dtype)
    if spike is not None:                                         # shared direction of all queries and of one key
        q = (q * 0.2).to(dtype)
        q[:, :, 0] = 4.0
        for k in keys:
            k[:, :, 0] = 0.0
        keys[spike[0]][spike[1], :, 0] = 12.0 / (scale * 4.0)
        vals[spike[0]][spike[1]] = 5.0
    gate, sink = rnd(T, H + 3, seed=60, dtype=dtype), rnd(H, seed=61) + sink_at
    kc, vc, table = paged(keys, vals, page, dtype, device)
    wide = torch.full((T, H * dv + 24), 7.0, dtype=dtype, device=device)
    out = wide[:, 8:8 + H * dv]
    ops.paged_attention(q.to(device), kc, vc, table, i32(ctx, device), i32([0] + torch.tensor(lens).cumsum(0).tolist(), device),
                        max(lens), scale, window=window, max_ctx=max(ctx), keep_first=keep, sink=sink.to(device),
                        gate=gate.to(device)[:, 3:] if gated else None, out_scale=out_scale, out=out)
    assert bool((wide[:, :8] == 7).all()) and bool((wide[:, 8 + H * dv:] == 7).all())
    res, t = [], 0
    for i, n in enumerate(lens):
        mask = {"size": window if window else ctx[i] + 1, "keep_first": keep}
        want = oracle.sink_softmax(d(q)[t:t + n], d(keys[i]), d(vals[i]), scale, mask, d(sink)) * out_scale
        if gated:
            want = want * oracle.sigmoid(d(gate)[t:t + n, 3:])[:, :, None]
        res.append((out[t:t + n].reshape(n, H, dv), want))
        t += n
    status_ok(device)
    return res


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,G,dk,dv", SHAPES)
@pytest.mark.parametrize("window,keep", [(37, 3), (129, 70), (1, 1), (0, 0), (64, 0)])
def test_sink_attention_with_kept_first_tokens(device, dtype, H, G, dk, dv, window, keep):
    for lens, ctx in (([1, 1, 1], [5, 64, 300]), ([130, 1, 7], [130, 300, 70])):
        for got, want in run_attention(device, dtype, H, G, dk, dv, lens, ctx, window, keep):
            close(got, want, dtype, tol16=2e-2)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("window,keep,far", [(75, 3, 500), (64, 1, 320), (128, 130, 700), (200, 64, 513), (1, 2, 130)])
def test_edges_of_the_window_and_of_the_kept_tokens(device, dtype, window, keep, far):
    """One key stands out for every query: it must show just inside the window and among the kept first tokens, and be gone
    right behind either edge; as a single decoded token, as the last of a portion of two, and inside longer portions."""
    inside, outside = far - window, far - window - 1                       # (the query is position far - 1)
    places = {inside: True, outside: outside < keep, keep - 1: True, keep: keep >= inside, 0: True, far - 1: True}
    for at, seen in places.items():
        for lens in ([1], [2], [40], [1, 3]):
            ctx = [far] + [far - 7] * (len(lens) - 1)
            (got, want), *rest = run_attention(device, dtype, 4, 2, 32, 32, lens, ctx, window, keep, spike=(0, at), out_scale=1.0,
                                               gated=False)
            close(got, want, dtype, tol16=2e-2)
            share = float(d(got)[-1].mean())
            assert share > 4 if seen else share < 2, (at, seen, share)
            for g, w in rest:
                close(g, w, dtype, tol16=2e-2)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("sink_at", [-40.0, 3.0, 12.0, 60.0])
def test_sinks_of_any_size(device, dtype, sink_at):
    for lens, ctx in (([1, 1], [9, 400]), ([150, 2], [150, 400])):
        for got, want in run_attention(device, dtype, 4, 2, 64, 32, lens, ctx, 90, 5, sink_at=sink_at):
            assert torch.isfinite(got.float()).all()
            close(got, want, dtype, tol16=2e-2)


@gpu
@pytest.mark.parametrize("n_splits", [1, 2, 5, 9])
def test_decode_splits_with_kept_tiles(n_splits):
    """A sink counts once however the keys are split, and splits cover the kept tiles and the window's."""
    sm = ops.sm100
    for window, keep in ((300, 140), (1024, 4), (0, 0), (17, 260)):
        H, G, D, ctx = 8, 2, 64, [1100, 200, 513]
        keys, vals = [rnd(c, G, D, seed=i, dtype=torch.bfloat16) for i, c in enumerate(ctx)], [rnd(c, G, D, seed=9 + i, dtype=torch.bfloat16) for i, c in enumerate(ctx)]
        q, sink = rnd(3, H, D, seed=20, dtype=torch.bfloat16), rnd(H, seed=21) + 2
        kc, vc, table = paged(keys, vals, 64, torch.bfloat16, "cuda:0")
        got = sm.attention_ext(q.cuda(), kc, vc, table, i32(ctx, "cuda:0"), i32([0, 1, 2, 3], "cuda:0"), 1, 0.2, window, keep,
                               sink.cuda(), n_splits=n_splits)
        for i in range(3):
            want = oracle.sink_softmax(d(q)[i:i + 1], d(keys[i]), d(vals[i]), 0.2, {"size": window or 9999, "keep_first": keep}, d(sink))
            close(got[i].view(1, H, D), want, torch.bfloat16, tol16=2e-2)
    status_ok("cuda:0")


# ------------------------------------------------------------------------------------------- HGRN2
def forget_case(dtype, H, N, P, lens, seed=0, kind="spread"):
    """Projections of sequences of ``lens`` tokens, bias and lower bounds. ``kind``: gates spread from closed to open; all
    nearly open (long memories); or closed now and then (products of gates underflow)."""
    qs, fs, vs = ([rnd(n, w, seed=seed + s * 100 + i, dtype=dtype) for i, n in enumerate(lens)] for s, w in
                  ((1, H * N), (2, H * N), (3, H * P)))
    u = torch.rand(H * N, generator=torch.Generator().manual_seed(seed))
    b, lower = {"spread": (8 * u - 2, (u - 0.3).clamp(min=0)), "open": (6 + 6 * u, 0.5 * u),
                "closed": (4 * u, torch.zeros(H * N))}[kind]
    if kind == "closed":
        for f in fs:
            f[::5] = -200.0
    return qs, fs, vs, b, lower, 1 + rnd(P, seed=seed + 7, k=0.2)


def forget_expected(q, f, v, b, lower, nw, H, N, P, eps, scale, S=None):
    T = q.shape[0]
    keep = oracle.forget(d(f) + d(b), d(lower)).view(T, H, N)
    o, S = oracle.forget_write(oracle.silu(d(q)).view(T, H, N), keep, d(v).view(T, H, P), S)
    return (oracle.rms(o, eps) * d(nw) * scale).reshape(T, H * P), S


HEADS = [(3, 40, 56), (2, 13, 19), (2, 128, 128), (4, 64, 64), (1, 130, 3), (2, 72, 24), (1, 48, 136), (2, 8, 128), (3, 20, 7), (1, 300, 40)]
LENS = [1, 70, 33, 200]
CUTS = {"whole": [[300]] * 4, "tokens": [[1]] * 4, "twos": [[2]] * 4,
        "mixed": [[1], [5, 1, 2, 40], [17, 16], [9, 64, 1, 2, 8, 7, 100]]}


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,N,P,cuts", [(*s, c) for s in HEADS for c in ("whole", "mixed")]
                         + [(*s, c) for s in HEADS[:4] for c in ("tokens", "twos")])
def test_forget_scan_in_portions(device, dtype, H, N, P, cuts):
    """Unequal sequences in portions of every size, states in slots that others used, outputs beside other columns."""
    eps, scale = 1e-5, 0.8
    qs, fs, vs, b, lower, nw = forget_case(dtype, H, N, P, LENS)
    want = [forget_expected(q, f, v, b, lower, nw, H, N, P, eps, scale) for q, f, v in zip(qs, fs, vs)]
    slots = [4, 1, 5, 2]
    state = rnd(6, H, P, N, seed=77).to(device)
    before = state.clone()
    state[slots] = 0
    got = [[] for _ in LENS]
    dev = lambda t: t.to(device)                                            # noqa: E731
    for step in portions(LENS, CUTS[cuts]):
        cat = lambda xs: torch.cat([xs[i][t:t + c] for i, t, c in step])    # noqa: E731
        proj = torch.cat([cat(qs), cat(fs), cat(vs), torch.zeros(sum(c for _, _, c in step), (-H * (2 * N + P)) % 8, dtype=dtype)], 1)
        proj, cu = dev(proj), bounds(step, device)
        wide = torch.full((proj.shape[0], H * P + 8), 3.0, dtype=dtype, device=device)
        out = ops.forget_scan(proj[:, :H * N], proj[:, H * N:2 * H * N], proj[:, 2 * H * N:H * (2 * N + P)], dev(b), dev(lower), state, cu,
                              i32([slots[i] for i, _, _ in step], device), H, N, P, dev(nw), eps, scale,
                              max_len=max(c for _, _, c in step), cu_host=cu.tolist(), out=wide[:, 8:])
        assert bool((wide[:, :8] == 3).all())
        for j, (i, _, _) in enumerate(step):
            got[i].append(out[cu[j]:cu[j + 1]].clone())
    for i in range(len(LENS)):
        close(torch.cat(got[i]), want[i][0], dtype, 5e-5, 2e-2)
        close(state[slots[i]].transpose(1, 2), want[i][1], dtype, 2e-5, 2e-3)
    assert torch.equal(state[[0, 3]], before[[0, 3]])
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("kind", ["open", "closed"])
@pytest.mark.parametrize("H,N,P", [(2, 128, 128), (3, 48, 64), (2, 64, 40)])
def test_forget_scan_with_long_memories_and_closed_gates(device, dtype, kind, H, N, P):
    """Gates near 1 over several chunks, where 1 - F is small and the state keeps every token, and gates that are exactly 0
    every few tokens, where products of gates vanish."""
    n, eps = 700, 1e-5
    (q,), (f,), (v,), b, lower, nw = forget_case(dtype, H, N, P, [n], 5, kind)
    want, S = forget_expected(q, f, v, b, lower, nw, H, N, P, eps, 1.0)
    dev = lambda t: t.to(device)                                            # noqa: E731
    for cuts in ([n], [256, 1, 130, 2, n - 389]):
        state, at = torch.zeros(1, H, P, N, device=device), 0
        for c in cuts:
            s = slice(at, at + c)
            out = ops.forget_scan(dev(q[s]), dev(f[s]), dev(v[s]), dev(b), dev(lower), state, i32([0, c], device), i32([0], device), H, N, P,
                                  dev(nw), eps, 1.0, max_len=c, cu_host=[0, c])
            assert torch.isfinite(out.float()).all()
            close(out, want[s], dtype, 2e-4, 2e-2)
            at += c
        close(state[0].transpose(1, 2), S, dtype, 1e-4, 2e-3)
    status_ok(device)


@gpu
@pytest.mark.parametrize("H,N,P", [(2, 128, 128), (2, 40, 24), (1, 64, 100), (1, 96, 64)])
def test_single_writes_show_at_every_distance(H, N, P):
    """Only one token writes; it must reach every later token of its chunk and of later ones with the product of the gates
    between them, and none before it: every pair of places inside a chunk's blocks is covered by some choice."""
    dt, dev, eps = torch.bfloat16, "cuda:0", 1e-12
    n = 150
    (q,), (f,), (v,), b, lower, nw = forget_case(dt, H, N, P, [n], 11)
    for at in (0, 5, 7, 8, 15, 16, 31, 33, 63, 64, 65, 100, 127, 128, 140):
        one = torch.zeros_like(v)
        one[at] = v[at]
        keep = oracle.forget(d(f) + d(b), d(lower)).view(n, H, N)
        o, _ = oracle.forget_write(oracle.silu(d(q)).view(n, H, N), keep, d(one).view(n, H, P))
        state = torch.zeros(1, H, P, N, device=dev)
        out = ops.sm100.forget_scan(q.to(dev), f.to(dev), one.to(dev), b.to(dev), lower.to(dev), state, i32([0, n], dev), i32([0], dev),
                                    H, N, P, torch.ones(P, device=dev), eps, 1.0, max_len=n, cu_host=[0, n], chunked=True)
        assert not out[:at].any()
        want = oracle.rms(o, eps).reshape(n, H * P)
        far = (o.pow(2).mean(-1) > 1e-6).repeat_interleave(P, 1)                 # what is not lost in rounding
        close(torch.where(far, d(out), 0.0), torch.where(far, want, 0.0), dt, tol16=4e-2)
    status_ok(dev)


# ------------------------------------------------------------------------------------------- residual, gates, depth average
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("W", [64, 90, 2048, 5000])
@pytest.mark.parametrize("T", [1, 37, 400])
def test_gated_residual_and_depth_average(device, dtype, W, T):
    eps, L = 1e-5, 10
    dev = lambda t: t.to(device)                                            # noqa: E731
    emb = rnd(40, W, seed=1, dtype=dtype)
    ids = torch.randint(0, 40, (T,), generator=torch.Generator().manual_seed(2)).int()
    n0 = rnd(W, seed=3, k=0.3)
    for average, gated in ((True, True), (True, False), (False, True)):
        x, hist, h = ops.depth_start(dev(emb), dev(ids), L, dev(n0), eps, 1.0, average)
        wx = d(emb)[ids.long()]
        outputs, all_coef = [wx], [rnd(i + 2, seed=60 + i, k=0.6) for i in range(L)]
        assert (hist is not None) == average
        close(h, oracle.model_norm(wx, d(n0), eps), dtype)
        for i in range(L):
            proj = rnd(T, 2 * W + 24, seed=10 + i, dtype=dtype)
            y1, y2, bias = rnd(T, W, seed=20 + i, dtype=dtype), rnd(T, W, seed=30 + i, dtype=dtype), rnd(W, seed=40 + i)
            gb, coef, nw = rnd(2 * W, seed=50 + i), all_coef[i], rnd(W, seed=70 + i, k=0.3)
            has_ff, has_bias, last = i != 2, i % 2 == 0, i + 1 == L
            rows = torch.tensor([T - 1, 0, T - 1]) if last else None
            g1, g2 = proj[:, 8:8 + W], proj[:, 16 + W:16 + 2 * W]
            pd = dev(proj)
            y2_dev = dev(y2)
            want = d(y1)
            ff = d(y2) + (d(bias) if has_bias else 0)
            if device != "cpu" and i == 1:                                   # expert rows that are still to be summed
                parts = rnd(T * 3, W, seed=80, dtype=dtype)
                y2_dev, ff = ops.sm100.PendingCombine(dev(parts), torch.zeros(T, 3, dtype=torch.int32), 0, 4, None, T, W, 3), d(parts).view(T, 3, W).sum(1)
            if gated:
                want, ff = want * oracle.sigmoid(d(g1) + d(gb)[:W]), ff * oracle.sigmoid(d(g2) + d(gb)[W:])
            wx = wx + want + (ff if has_ff else 0)
            outputs.append(wx)
            if average:
                wx = oracle.depth_average(d(coef), outputs)
            x, h = ops.depth_step(x, hist, i, dev(y1), pd[:, 8:8 + W] if gated else None, dev(gb)[:W] if gated else None,
                                  y2_dev if has_ff else None, pd[:, 16 + W:16 + 2 * W] if gated and has_ff else None,
                                  dev(gb)[W:] if gated and has_ff else None, dev(bias) if has_bias else None,
                                  [dev(c) for c in all_coef[i:i + 4]] if average else None, dev(nw), eps, 1.0, dev(rows) if last else None)
            if last:
                wx = wx[rows]
            close(x, wx, torch.float32, 5e-6 if dtype == torch.float32 else 5e-5)
            close(h, oracle.model_norm(wx, d(nw), eps), dtype)


# ------------------------------------------------------------------------------------------- feed-forward parts
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,K,ff", [(1, 64, 96), (5, 2048, 512), (300, 256, 200), (33, 90, 27), (70, 128, 1000)])
def test_biases_of_the_gated_feed_forward_part(device, dtype, T, K, ff):
    x, wg, wu = rnd(T, K, seed=1, dtype=dtype), rnd(ff, K, seed=2, dtype=dtype, k=K ** -0.5), rnd(ff, K, seed=3, dtype=dtype, k=K ** -0.5)
    b = rnd(2 * ff, seed=4)
    want = oracle.silu(d(x) @ d(wg).T + d(b)[:ff]) * (d(x) @ d(wu).T + d(b)[ff:])
    close(ops.gate_up_act(x.to(device), torch.cat([wg, wu]).to(device), ff, "silu", b.to(device)), want, dtype)
    if device == "cuda:0" and dtype == torch.bfloat16 and K % 8 == 0 and ff % 8 == 0:
        for sk in (1, 2):                                                    # also where the product is split
            close(ops.sm100.gate_up_act(x.to(device), torch.cat([wg, wu]).to(device), ff, split_k=sk, bias=b.to(device)), want, dtype)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,W,ff,E,top", [(t, *s) for t in (1, 13, 64, 65, 200) for s in (
    (96, 56, 6, 3), (256, 64, 8, 2), (90, 27, 3, 1), (64, 40, 4, 4))] + [(1, 4096, 16, 140, 6), (13, 4096, 16, 140, 6)])
def test_experts_behind_a_router_with_a_logit_bias(device, dtype, T, W, ff, E, top):
    """Through the model's own feed-forward function. The bias decides choices (some experts lead by it alone) and weights."""
    from legion_b200.models.decoder import Decoder
    x = rnd(T, W, seed=1, dtype=dtype)
    ow = {"m.router": rnd(E, W, seed=2, dtype=dtype, k=2 * W ** -0.5), "m.router.b": rnd(E, seed=3, k=2.0)}
    for e in range(E):
        for n, o, k in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
            ow[f"m.e{e}.{n}"] = rnd(o, k, seed=len(ow) + 5, dtype=dtype, k=k ** -0.5)
    w64 = {k: d(v) for k, v in ow.items()}
    want = oracle.moe(d(x), w64, "m", {"router": {"top": top}})
    z = d(x) @ w64["m.router"].T + w64["m.router.b"]
    if E > 1:
        assert (z.topk(top).indices.sort().values != (z - w64["m.router.b"]).topk(top).indices.sort().values).any() or top == E
    dec = Decoder.__new__(Decoder)
    dec.cfg = ModelConfig(arch="mananex", hidden=W, vocab=8, parallel_sublayers=True,
                          layers=[LayerSpec(SsdSpec(1, 8, 8), MoeSpec(E, top, ff, router="biased_softmax"))])
    dec.w = {"l0.moe.router": ow["m.router"], "l0.moe.router_bias": ow["m.router.b"],
             "l0.moe.gate_up": torch.stack([torch.cat([ow[f"m.e{e}.gate"], ow[f"m.e{e}.up"]]) for e in range(E)]),
             "l0.moe.down": torch.stack([ow[f"m.e{e}.down"] for e in range(E)])}
    dec.w = {k: v.to(device) for k, v in dec.w.items()}
    dec._shared_down = {}
    s = z.sort(-1, descending=True).values
    clear = torch.ones(T, dtype=torch.bool) if top == E else s[:, top - 1] - s[:, top] > 1e-4       # no choice hangs on rounding
    for _ in range(2):
        y = dec._spec_ffn("l0", 0, x.to(device))[0][0]
        got, _ = ops.depth_step(torch.zeros(T, W, device=device), None, 0, torch.zeros(T, W, dtype=dtype, device=device), None, None, y,
                                None, None, None, None, torch.zeros(W, device=device), 1e-5, 1.0)
        close(got.cpu()[clear], want[clear], dtype, 2e-5, 2e-2)
    ids, wts = ops.router(x.to(device), dec.w["l0.moe.router"], top, "biased_softmax", True, 1.0, dec.w["l0.moe.router_bias"], n_local=E)
    for t in range(T):
        if clear[t]:
            r = oracle.route(z[t], top)
            assert {int(e) for e in ids[t]} == set(r)
            assert all(math.isclose(float(c), float(r[int(e)]), rel_tol=1e-3, abs_tol=1e-4) for e, c in zip(ids[t], wts[t]))
    status_ok(device)


def test_biased_dense_specification_is_the_parallel_form_only():
    with pytest.raises(ValueError):
        ModelConfig(layers=[LayerSpec(SsdSpec(1, 8, 8), DenseSpec(8, bias=True))])
