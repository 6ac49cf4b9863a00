"""Each mechanism of the Gurozen design alone, against the functions of ``gurozen_oracle`` (float64): on CPU the reference
ops, on a GPU the kernels in fp32 and bf16."""
import math

import pytest
import torch

import gurozen_oracle as oracle
from legion_b200 import ops
from legion_b200.config import LayerSpec, LoopSpec, ModelConfig, PRESETS, RotarySpec

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


LENS = [1, 70, 33, 130]
CUTS = {"whole": [[200]] * 4, "tokens": [[1]] * 4, "twos": [[2]] * 4,
        "mixed": [[1], [5, 1, 2, 40], [17, 16], [9, 64, 1, 2, 8, 7]]}
SLOTS = [4, 1, 5, 2]


# ------------------------------------------------------------------------------------------- residual and norms
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("W", [64, 90, 2048, 131])
@pytest.mark.parametrize("T", [1, 37])
def test_prenorm_steps(device, dtype, W, T):
    """Start with and without a norm of the embedding rows, two terms, a term of several rows, and only the norm."""
    eps, m, V = 1e-5, 0.6, 40
    emb, pre, n1 = rnd(V, W, seed=1, dtype=dtype), rnd(W, seed=2, k=0.3), rnd(W, seed=3, k=0.3)
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(4)).int()
    dev = lambda t: t.to(device)                                            # noqa: E731
    both = torch.zeros(T, 2 * W, dtype=dtype, device=device)
    x0 = oracle.model_norm(d(emb)[ids.long()], d(pre), eps)
    x, h = ops.prenorm_start(dev(emb), dev(ids), dev(pre), dev(n1), eps, 1.0, raw=both[:, W:])
    close(x, x0, torch.float32)
    close(h, oracle.model_norm(x0, d(n1), eps), dtype)
    close(both[:, W:], x0, dtype)
    assert not both[:, :W].any()
    xr, none = ops.prenorm_start(dev(emb)[:T] if T <= V else None, None, None, None, eps, 1.0, raw=both[:, :W])
    assert none is None
    close(xr, d(emb)[:T], torch.float32, 1e-7)
    y, y1 = rnd(T, W, seed=5, dtype=dtype, k=2.0), rnd(T, W, seed=6, dtype=dtype)
    want = x0 + m * (d(y) + 0.5 * d(y1))
    x, h = ops.prenorm_step(x, [(dev(y), 1.0), (dev(y1), 0.5)], m, dev(n1), eps, 1.0, dtype=dtype)
    close(x, want, torch.float32)
    close(h, oracle.model_norm(want, d(n1), eps), dtype)
    x, h = ops.prenorm_step(x, [(dev(y), 1.0)], m, None, eps, 1.0, raw=both[:, :W], dtype=dtype)
    want = want + m * d(y)
    assert h is None
    close(x, want, torch.float32)
    close(both[:, :W], want, dtype)
    x2, h = ops.prenorm_step(x, (), 1.0, dev(n1), eps, 1.0, dtype=dtype)
    close(x2, want, torch.float32)
    close(h, oracle.model_norm(want, d(n1), eps), dtype)
    if device != "cpu":
        rows = rnd(T * 3, W, seed=7, dtype=dtype)
        p = ops.sm100.PendingCombine(dev(rows), torch.zeros(T, 2, dtype=torch.int32), 0, 3, None, T, W, 3)
        x, h = ops.prenorm_step(x, [(p, 1.0), (dev(y1), 1.0)], m, dev(n1), eps, 1.0, dtype=dtype)
        close(x, want + m * (d(rows).view(T, 3, W).sum(1) + d(y1)), torch.float32)


# ------------------------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("dims,base,factor,low,high,original", [
    (64, 1e4, 4.0, 1.0, 4.0, 96), (128, 5e5, 8.0, 1.0, 4.0, 8192), (10, 3e3, 2.0, 1.0, 2.0, 40), (2, 1e4, 4.0, 1.0, 4.0, 64),
    (32, 1e4, 1.0, 1.0, 4.0, 256), (24, 1e2, 16.0, 2.0, 16.0, 500)])
def test_rotation_frequencies(dims, base, factor, low, high, original):
    r = RotarySpec(dims, base, factor, original, scaling="llama3", low=low, high=high, layout="half")
    from legion_b200.models.decoder import Decoder
    dec = Decoder.__new__(Decoder)
    dec._rot, dec.device = {}, torch.device("cpu")
    table = dec.rotary_table(r, 400)
    f = oracle.frequencies({"dims": dims, "base": base, "scaling": dict(factor=factor, low=low, high=high, original=original)})
    ang = torch.arange(400, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    assert float((table.double() - torch.cat([ang.cos(), ang.sin()], 1)).abs().max()) < 1e-6
    plain = dec.rotary_table(RotarySpec(dims, base, layout="half"), 400)
    ang = torch.arange(400, dtype=torch.float64)[:, None] * torch.tensor(oracle.frequencies({"dims": dims, "base": base}), dtype=torch.float64)
    assert float((plain.double() - torch.cat([ang.cos(), ang.sin()], 1)).abs().max()) < 1e-6


# ------------------------------------------------------------------------------------------- q, k, v in front of the scores
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,G,dk,dv,K,dims", [(6, 2, 40, 56, 4, 24), (1, 1, 21, 11, 1, 10), (8, 2, 128, 64, 3, 128),
                                              (3, 3, 64, 32, 2, 64), (3, 1, 17, 35, 6, 2), (2, 1, 16, 8, 9, 16)])
def test_projected_rows_on_their_way_to_the_cache(device, dtype, H, G, dk, dv, K, dims):
    """Bias, short convolution with carried history, norm over the whole of q and of k, rotation, append; portions of every
    size. Cells and slots of others stay as they are."""
    C, nq, nk = (H + G) * dk + G * dv, H * dk, G * dk
    xs = [rnd(n, C, seed=n, dtype=dtype) for n in LENS]
    b, w = rnd(C, seed=1, k=0.5), rnd(C, K, seed=2, k=0.6)
    qn, kn = 1 + rnd(nq, seed=3, k=0.3), 1 + rnd(nk, seed=4, k=0.3)
    rot = {"dims": dims, "base": 50.0}
    f = oracle.frequencies(rot)
    want = []
    for x in xs:
        u = oracle.short_conv(d(x) + d(b), d(w))
        q = (oracle.rms(u[:, :nq], 1e-5) * d(qn)).view(-1, H, dk)
        k = (oracle.rms(u[:, nq:nq + nk], 1e-5) * d(kn)).view(-1, G, dk)
        pos = range(x.shape[0])
        want.append((oracle.rotate(q, pos, rot), oracle.rotate(k, pos, rot), u[:, nq + nk:].view(-1, G, dv)))
    ang = torch.arange(256, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    cs = torch.cat([ang.cos(), ang.sin()], 1).float().to(device)
    dev = lambda t: t.to(device)                                            # noqa: E731
    page = 16
    for name, cuts in CUTS.items():
        kc = torch.full((60, page, G, dk), 7.0, dtype=dtype, device=device)
        vc = torch.full((60, page, G, dv), 7.0, dtype=dtype, device=device)
        hist = torch.full((6, K - 1, C), 9.0, device=device)
        hist[SLOTS] = 0.0
        cell = lambda i, t: (i * 13 + 3) * page + t                         # noqa: E731
        got = [[] for _ in LENS]
        for step in portions(LENS, cuts):
            x = dev(torch.cat([xs[i][a:a + c] for i, a, c in step]))
            pos = i32([t for _, a, c in step for t in range(a, a + c)], device)
            slots = torch.tensor([cell(i, t) for i, a, c in step for t in range(a, a + c)], device=device)
            q = ops.qkv_conv_append(x, dev(b), dev(w.t().contiguous()), hist if K > 1 else None, bounds(step, device),
                                    i32([SLOTS[i] for i, _, _ in step], device), dev(qn), dev(kn), "all", 1e-5, cs, "half", pos,
                                    slots, kc, vc, H, max_len=max(c for _, _, c in step))
            at = 0
            for i, _, c in step:
                got[i].append(q[at:at + c])
                at += c
        for i, n in enumerate(LENS):
            close(torch.cat(got[i]), want[i][0], dtype)
            rows = [cell(i, t) for t in range(n)]
            close(kc.view(-1, G, dk)[rows], want[i][1], dtype)
            close(vc.view(-1, G, dv)[rows], want[i][2], dtype)
            if K > 1 and n >= K - 1:
                close(hist[SLOTS[i]], (d(xs[i]) + d(b))[n - K + 1:], torch.float32)
        used = torch.zeros(60 * page, dtype=torch.bool)
        used[[cell(i, t) for i, n in enumerate(LENS) for t in range(n)]] = True
        assert bool((kc.view(-1, G, dk)[~used.to(device)] == 7).all()) and bool((vc.view(-1, G, dv)[~used.to(device)] == 7).all())
        assert bool((hist[[0, 3]] == 9.0).all()), name


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("layout", ["half", "pairs"])
def test_projected_rows_with_other_options(device, dtype, layout):
    """Norms of each head, no bias, no convolution, either rotation; a padding row writes no cell; nothing kept of a step
    that must not write its state."""
    H, G, dk, dv, T = 4, 2, 32, 24, 9
    x = rnd(T, (H + G) * dk + G * dv, seed=1, dtype=dtype)
    qn, kn = 1 + rnd(dk, seed=3, k=0.3), 1 + rnd(dk, seed=4, k=0.3)
    ang = torch.arange(64, dtype=torch.float64)[:, None] * torch.tensor([0.3, 0.05, 1.0, 0.7])
    cs = torch.cat([ang.cos(), ang.sin()], 1).float()
    q = oracle.rms(d(x)[:, :H * dk].view(T, H, dk), 1e-5) * d(qn)
    want = q.clone()
    for i in range(4):
        a, z = (i, i + 4) if layout == "half" else (2 * i, 2 * i + 1)
        c, s = ang.cos()[5:5 + T, i, None], ang.sin()[5:5 + T, i, None]
        want[..., a], want[..., z] = q[..., a] * c - q[..., z] * s, q[..., z] * c + q[..., a] * s
    kc, vc = (torch.zeros(4, 16, G, n, dtype=dtype, device=device) for n in (dk, dv))
    slots = torch.arange(T, device=device) + 20
    slots[3] = -1
    dev = lambda t: t.to(device)                                            # noqa: E731
    got = ops.qkv_conv_append(dev(x), None, None, None, i32([0, T], device), i32([0], device), dev(qn), dev(kn), "head", 1e-5,
                              dev(cs), layout, i32(range(5, 5 + T), device), slots, kc, vc, H, max_len=T)
    close(got, want, dtype)
    live = [20 + i for i in range(T) if i != 3]
    close(vc.view(-1, G, dv)[live], d(x)[[i for i in range(T) if i != 3], (H + G) * dk:].view(-1, G, dv), dtype)
    assert not vc.view(-1, G, dv)[23].any() and not kc.view(-1, G, dk)[23].any()
    hist = rnd(2, 2, x.shape[1], seed=8, device=device)
    keep = hist.clone()
    for n in (1, 5):
        ops.qkv_conv_append(dev(x)[:n], None, rnd(3, x.shape[1], seed=9, device=device), hist, i32([0, n], device), i32([1], device),
                            None, None, "all", 1e-5, None, "half", i32(range(n), device), slots[:n], kc, vc, H, write_state=False,
                            max_len=n)
    assert torch.equal(hist, keep)


# ------------------------------------------------------------------------------------------- soft-capped attention
def paged(k, v, page, device, dtype, order):
    n = -(-k.shape[0] // page)
    kc = torch.full((n + 2, page, *k.shape[1:]), 3.0)
    vc = torch.full((n + 2, page, *v.shape[1:]), 3.0)
    table = [order[i % len(order)] if len(order) == n else n + 1 - i for i in range(n)]
    for t in range(k.shape[0]):
        kc[table[t // page], t % page], vc[table[t // page], t % page] = k[t], v[t]
    return kc.to(dtype).to(device), vc.to(dtype).to(device), i32([table], device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 128, 128), (6, 3, 40, 72), (1, 1, 64, 64), (3, 1, 136, 24), (2, 1, 13, 19), (18, 1, 96, 160),
                                       (2, 2, 256, 256)])
@pytest.mark.parametrize("cap", [3.0, 30.0])
def test_soft_capped_attention_prompts_and_decode(device, dtype, H, G, dk, dv, cap):
    n, scale = 300, 1.5 * dk ** -0.5
    q, k, v = rnd(n, H, dk, seed=1, dtype=dtype, k=2.0), rnd(n, G, dk, seed=2, dtype=dtype, k=2.0), rnd(n, G, dv, seed=3, dtype=dtype)
    want = oracle.softmax_heads(d(q), d(k), d(v), scale, cap)
    assert float((want - oracle.softmax_heads(d(q), d(k), d(v), scale)).abs().max()) > 1e-2       # the cap matters
    kc, vc, bt = paged(k, v, 64, device, dtype, [])
    for a, z in ((0, n), (0, 65), (200, 202), (n - 1, n), (63, 64), (100, 230)):
        o = ops.paged_attention(q[a:z].contiguous().to(device), kc, vc, bt, i32([z], device), i32([0, z - a], device), z - a, scale,
                                max_ctx=z, softcap=cap)
        close(o, want[a:z], dtype, 2e-5, 2e-2)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("far", [0, 63, 64, 127, 128, 511])
def test_one_far_key_under_the_cap(device, dtype, far):
    """A key that stands out by far more than the cap: it weighs e^(2 cap) against the others and no more."""
    n, H, G, dk, dv, cap = 700, 4, 2, 64, 32, 4.0
    q, k, v = rnd(n, H, dk, seed=1, dtype=dtype, k=0.05), rnd(n, G, dk, seed=2, dtype=dtype, k=0.05), rnd(n, G, dv, seed=3, dtype=dtype)
    q[-3:, :, 0], k[:, :, 0], k[far, :, 0], v[far] = 20.0, -20.0, 20.0, 8.0
    want = oracle.softmax_heads(d(q), d(k), d(v), 0.125, cap)
    kc, vc, bt = paged(k, v, 64, device, dtype, [])
    for a in (n - 1, n - 3):
        o = ops.paged_attention(q[a:].contiguous().to(device), kc, vc, bt, i32([n], device), i32([0, n - a], device), n - a, 0.125,
                                max_ctx=n, softcap=cap)
        close(o, want[a:], dtype)
    assert float(want[-1].mean()) > 4.0                                     # most of the weight is on it, not all


# ------------------------------------------------------------------------------------------- delta rule
def delta_case(H, G, dk, dv, K, dtype, lens=LENS):
    """Inputs, weights, and per sequence the oracle's outputs and last states."""
    C = 2 * G * dk + H * dv
    xs = [rnd(n, C, seed=n, dtype=dtype) for n in lens]
    As = [rnd(n, H * dk, seed=100 + n, dtype=dtype) for n in lens]
    Bs = [rnd(n, H, seed=200 + n, dtype=dtype) for n in lens]
    w = rnd(C, K, seed=1, k=0.8)
    A_log = torch.log(0.02 + 2 * torch.rand(H, generator=torch.Generator().manual_seed(2)) ** 2)
    bias = 4 * torch.rand(H * dk, generator=torch.Generator().manual_seed(3)) - 4
    want = []
    for x, a, b in zip(xs, As, Bs):
        T = x.shape[0]
        u = oracle.silu(oracle.short_conv(d(x), d(w)))
        unit = lambda t: oracle.unit(t.reshape(T, G, dk)).repeat_interleave(H // G, 1)                       # noqa: E731
        q, k = unit(u[:, :G * dk]) * dk ** -0.5, unit(u[:, G * dk:2 * G * dk])
        want.append(oracle.delta_rule(q, k, u[:, 2 * G * dk:].reshape(T, H, dv), oracle.decay(d(a), d(A_log), d(bias), H),
                                      oracle.sigmoid(d(b))))
    return xs, As, Bs, w, -torch.exp(A_log), bias, want


DELTA = [(6, 3, 40, 24, 4), (2, 2, 128, 128, 4), (1, 1, 13, 19, 1), (4, 1, 64, 72, 2), (2, 2, 7, 5, 6), (2, 1, 192, 136, 3),
         (3, 3, 32, 16, 3), (1, 1, 250, 33, 4)]


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,G,dk,dv,K", DELTA)
def test_channel_delta_prompts_portions_and_decode(device, dtype, H, G, dk, dv, K):
    xs, As, Bs, w, A, bias, want = delta_case(H, G, dk, dv, K, dtype)
    dev = lambda t: t.to(device)                                            # noqa: E731
    C, wt = w.shape[0], w.t().contiguous()
    norm, eps = 1 + rnd(dv, seed=7, k=0.2), 1e-5
    gates = [rnd(n, H * dv, seed=300 + n, dtype=dtype) for n in LENS]
    for name, cuts in CUTS.items():
        hist, state = torch.full((6, K - 1, C), 9.0, device=device), torch.full((6, H, dv, dk), 9.0, device=device)
        hist[SLOTS], state[SLOTS] = 0.0, 0.0
        got = [[] for _ in LENS]
        for step in portions(LENS, cuts):
            cat = lambda ts: dev(torch.cat([ts[i][a:a + c] for i, a, c in step]))                            # noqa: E731
            wide = torch.cat([cat(xs), cat(Bs)], 1)                         # column slices of one projection
            ml = max(c for _, _, c in step)
            args = (wide[:, :C], dev(wt), hist, cat(As), dev(A), dev(bias), wide[:, C:], state, bounds(step, device),
                    i32([SLOTS[i] for i, _, _ in step], device), H, G, dk, dv)
            if ml == 1 and device != "cpu":
                y = ops.sm100.channel_delta_decode(*args, cat(gates), dev(norm), eps)
            else:
                o = ops.channel_delta(*args, max_len=ml)
                y = ops.head_norm_gate(o, cat(gates), dev(norm), eps, H)
            at = 0
            for i, _, c in step:
                got[i].append(y[at:at + c])
                at += c
        for i in range(len(LENS)):
            o, S = want[i]
            y = (oracle.rms(o, eps) * d(norm)).reshape(o.shape[0], -1) * oracle.sigmoid(d(gates[i]))
            close(torch.cat(got[i]), y, dtype, 1e-4, 2e-2)
            close(state[SLOTS[i]].transpose(1, 2), S, dtype, 2e-5, 2e-3)
        assert bool((state[[0, 3]] == 9.0).all()) and bool((hist[[0, 3]] == 9.0).all()), name
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_channel_delta_without_writing_the_state(device, dtype):
    H, G, dk, dv, K = 2, 1, 32, 24, 3
    xs, As, Bs, w, A, bias, want = delta_case(H, G, dk, dv, K, dtype, [30])
    dev = lambda t: t.to(device)                                            # noqa: E731
    hist, state = torch.zeros(2, K - 1, w.shape[0], device=device), torch.zeros(2, H, dv, dk, device=device)
    o = ops.channel_delta(dev(xs[0]), dev(w.t().contiguous()), hist, dev(As[0]), dev(A), dev(bias), dev(Bs[0]), state, i32([0, 30], device),
                          i32([1], device), H, G, dk, dv, write_state=False, max_len=30)
    close(o, want[0][0].reshape(30, -1), dtype)
    assert not state.any() and not hist.any()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,K", [(4, 2, 64, 48, 4), (2, 2, 128, 128, 3)])
def test_channel_delta_in_slices(dtype, H, G, dk, dv, K, monkeypatch):
    """A scratch that holds a fraction of the step's records: sequences go on from slice to slice, at any token."""
    lens = [150, 1, 333, 64, 7]
    xs, As, Bs, w, A, bias, want = delta_case(H, G, dk, dv, K, dtype, lens)
    dev = lambda t: t.cuda()                                                # noqa: E731
    ws = ops.sm100.Workspace.get(torch.device("cuda", torch.cuda.current_device()))
    for room in (1, 40 * 4 * ops.sm100.ext().channel_delta_record_floats(H, dk, dv, dtype == torch.float32)):
        monkeypatch.setattr(ops.sm100, "DELTA_SCRATCH", room)
        ws._cache.pop("channel_delta_rec", None)
        hist, state = torch.zeros(6, K - 1, w.shape[0]).cuda(), torch.zeros(6, H, dv, dk).cuda()
        cu = i32([0] + torch.tensor(lens).cumsum(0).tolist(), "cuda")
        o = ops.channel_delta(dev(torch.cat(xs)), dev(w.t().contiguous()), hist, dev(torch.cat(As)), dev(A), dev(bias), dev(torch.cat(Bs)), state, cu,
                              i32([3, 0, 5, 1, 2], "cuda"), H, G, dk, dv, max_len=333)
        for i, (s, n) in enumerate(zip((3, 0, 5, 1, 2), lens)):
            at = sum(lens[:i])
            close(o[at:at + n], want[i][0].reshape(n, -1), dtype)
            close(state[s].transpose(1, 2), want[i][1], dtype, 2e-5, 2e-3)
            if n >= K - 1:
                close(hist[s], d(xs[i])[n - K + 1:], torch.float32)
        ws._cache.pop("channel_delta_rec", None)
    status_ok("cuda:0")


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("raw,first", [(-20.0, 1.0), (3.0, 0.0), (60.0, 0.0)])
def test_channel_delta_slow_and_instant_decays(device, dtype, raw, first):
    """Decays of almost one keep a far write; decays of (almost) zero drop it at once, without an overflow anywhere in a
    block. One channel at a time is written and read."""
    dk, dv, n = 32, 16, 500
    x = torch.zeros(n, 2 * dk + dv)
    x[:, 0], x[:, dk + 1] = 40.0, 40.0                                      # q reads channel 0, k writes channel 1
    x[0, dk:2 * dk] = 0.0
    x[0, dk] = 40.0                                                         # but the first token writes channel 0
    x[:, 2 * dk:] = 2.0
    a, b = torch.full((n, dk), raw), torch.full((n, 1), 30.0)
    w = torch.ones(1, x.shape[1])
    dev = lambda t: t.to(dtype).to(device)                                  # noqa: E731
    state, hist = torch.zeros(1, 1, dv, dk, device=device), torch.zeros(1, 0, x.shape[1], device=device)
    out = []
    cuts = [400, 1, 1, 98]
    for c in range(len(cuts)):
        lo, hi = sum(cuts[:c]), sum(cuts[:c + 1])
        out.append(ops.channel_delta(dev(x[lo:hi]), w.to(device), hist, dev(a[lo:hi]), torch.full((1,), -1.0, device=device),
                                     torch.zeros(dk, device=device), dev(b[lo:hi]), state, i32([0, hi - lo], device), i32([0], device),
                                     1, 1, dk, dv, max_len=hi - lo))
    o = d(torch.cat(out)) / (2.0 / (1 + math.exp(-2.0)) * dk ** -0.5)
    assert torch.isfinite(o).all() and abs(float(o[0].mean()) - 1) < 1e-2
    assert abs(float(o[-1].mean()) - first) < 2e-2, float(o[-1].mean())


# ------------------------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T", [1, 40, 200])
@pytest.mark.parametrize("E,top,count,keep", [(10, 3, 5, 2), (8, 4, 2, 1), (4, 4, 1, 1), (1, 1, 1, 1), (64, 6, 8, 3), (6, 2, 6, 4)])
def test_router_by_sigmoid_and_groups(device, dtype, T, E, top, count, keep):
    W = 64
    x, w = rnd(T, W, seed=1, dtype=dtype), rnd(E + 1, W, seed=2, dtype=dtype, k=1.5 / 8)
    w[:, 0] -= 0.4                                                          # small scores too
    x[:, 0] = 16.0
    r = ops.router(x.to(device), w.to(device), top, "sigmoid", "sum", 2.5, None, count, keep, n_local=E, group_top=2, gate_row=True,
                   shared_slots=2)
    ids, wts = r
    for t in range(T):
        z = (d(w) @ d(x[t]))
        want = oracle.route(z[:E], {"top": top, "scale": 2.5, "groups": {"count": count, "keep": keep}})
        got = dict(zip(ids[t].tolist(), wts[t].tolist()))
        assert set(got) == set(want) and all(abs(got[e] - float(want[e])) < 2e-5 for e in want), (got, want)
        if r.gate is not None:
            assert abs(float(r.gate[t]) - float(oracle.sigmoid(z[E]))) < 1e-5
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_router_weights_of_tiny_scores(device, dtype):
    """Scores whose sum is far below the floor that other routers hold it at."""
    x, w = torch.full((3, 64), 1.0, dtype=dtype, device=device), torch.full((4, 64), -0.5, dtype=dtype, device=device)
    w[1] *= 0.9375
    for T in (1, 3):
        ids, wts = ops.router(x[:T].repeat(40, 1) if T == 3 else x[:T], w, 2, "sigmoid", "sum", 1.0)
        assert ids[0].tolist()[0] == 1 and abs(float(wts[0].sum()) - 1) < 1e-4 and float(wts[0, 0]) > 0.8


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T", [1, 40, 150])
@pytest.mark.parametrize("W,ff,E,top,shared", [(96, 56, 6, 3, 72), (256, 64, 8, 2, 256), (90, 27, 3, 1, 27), (64, 40, 4, 4, 24), (128, 33, 4, 2, 70)])
def test_square_relu_experts_with_a_gated_shared_one(device, dtype, T, W, ff, E, top, shared):
    """Through the model's own feed-forward function: grouped products, the shared expert as slots of them (decode-sized
    steps) or as a part of its own (prompts), summed by the residual step."""
    from legion_b200.config import MoeSpec, SsdSpec
    from legion_b200.models.decoder import Decoder
    f = {"kind": "moe", "router": {"experts": E, "top": top, "scale": 1.5, "groups": {"count": 1, "keep": 1}}, "shared": {"ff": shared}}
    x = rnd(T, W, seed=1, dtype=dtype)
    ow = {"m.router": rnd(E, W, seed=2, dtype=dtype, k=2 * W ** -0.5), "m.shared.sg": rnd(1, W, seed=3, dtype=dtype, k=2 * W ** -0.5)}
    for n, width in [(f"e{e}", ff) for e in range(E)] + [("shared", shared)]:
        ow[f"m.{n}.up"], ow[f"m.{n}.down"] = rnd(width, W, seed=len(ow), dtype=dtype, k=W ** -0.5), rnd(W, width, seed=50 + len(ow), dtype=dtype, k=width ** -0.5)
    want = oracle.moe(d(x), {k: d(v) for k, v in ow.items()}, "m", f)
    spec = MoeSpec(E, top, ff, "relu2", router="sigmoid", renorm="sum", scale=1.5, shared_ff=shared, shared_gate=True)
    n = spec.shared_slots()
    assert n * ff >= shared > (n - 1) * ff
    up, down = torch.zeros(E + n, ff, W, dtype=dtype), torch.zeros(E + n, W, ff, dtype=dtype)
    for e in range(E):
        up[e], down[e] = ow[f"m.e{e}.up"], ow[f"m.e{e}.down"]
    up[E:].view(n * ff, W)[:shared] = ow["m.shared.up"]
    for j in range(n):
        c = min(ff, shared - j * ff)
        down[E + j, :, :c] = ow["m.shared.down"][:, j * ff:j * ff + c]
    dec = Decoder.__new__(Decoder)
    dec.cfg = ModelConfig(arch="gurozen", hidden=W, vocab=8, layers=[LayerSpec(SsdSpec(1, 8, 8), spec)])
    dec.w = {"l0.moe.router": torch.cat([ow["m.router"], ow["m.shared.sg"]]).to(device), "l0.moe.gate_up": up.to(device),
             "l0.moe.down": down.to(device)}
    dec._shared_down = {}
    for _ in range(2):
        terms = dec._spec_ffn("l0", 0, x.to(device))
        x0 = torch.zeros(T, W, device=device)
        y, _ = ops.prenorm_step(x0, terms, 1.0, torch.zeros(W, device=device), 1e-5, 1.0, dtype=dtype)
        close(y, want, dtype, 2e-5, 2e-2)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,K,N", [(1, 64, 96), (5, 2048, 512), (300, 256, 200), (33, 90, 27)])
def test_square_relu_and_row_factors_in_the_projection(device, dtype, T, K, N):
    x, w, s = rnd(T, K, seed=1, dtype=dtype), rnd(N, K, seed=2, dtype=dtype, k=K ** -0.5), rnd(T, seed=3)
    z = d(x) @ d(w).T
    close(ops.up_relu2(x.to(device), w.to(device)), torch.clamp(z, min=0) ** 2, dtype)
    close(ops.linear(x.to(device), w.to(device), tok_scale=s.to(device)), z * d(s)[:, None], dtype)
    close(ops.linear(x.to(device), w.to(device), out_dtype=torch.float32, tok_scale=s.to(device)), z * d(s)[:, None], torch.float32, 2e-4)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,n0,n1,rank", [(1, 64, 64, 8), (70, 96, 40, 24), (33, 128, 128, 16), (5, 21, 21, 8)])
def test_two_low_rank_products(device, dtype, T, n0, n1, rank):
    x, w = rnd(T, 16 + 2 * rank, seed=1, dtype=dtype), rnd(n0 + n1, rank, seed=2, dtype=dtype)
    a, g = ops.low_rank_pair(x.to(device)[:, 16:], w.to(device), n0, rank)
    close(a, d(x)[:, 16:16 + rank] @ d(w)[:n0].T, dtype)
    close(g, d(x)[:, 16 + rank:] @ d(w)[n0:].T, dtype)


# ------------------------------------------------------------------------------------------- layer runs
def test_runs_of_a_loop():
    c = PRESETS["tiny-gurozen"]()
    names = {k.split(".")[0] for k in __import__("legion_b200.models.weights", fromlist=["x"]).weight_shapes(c) if k[0] == "l" and k[1].isdigit()}
    assert len(names) == 1 + max(c.weight_layer(i) for i in range(c.n_layer)) < c.n_layer
    for start, stop, times, n in ((0, 2, 3, 4), (1, 4, 2, 4), (1, 2, 1, 2), (0, 1, 2, 1)):
        raw = list(range(n))
        lo = LoopSpec(start, stop, times)
        c.layers, c.loop = lo.expand(raw), lo
        runs = oracle.runs({"layers": raw, "loop": {"start": start, "stop": stop, "times": times}})
        assert [(c.weight_layer(i), c.begins_pass(i)) for i in range(len(c.layers))] == runs and c.layers == [i for i, _ in runs]
