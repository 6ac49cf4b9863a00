"""Each mechanism of the Pemezen design alone, against the functions of ``pemezen_oracle`` (float64): on CPU the reference
ops, on a GPU the kernels in fp32 and bf16."""
import math

import pytest
import torch

import pemezen_oracle as oracle
from legion_b200 import ops
from legion_b200.config import RotarySpec

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


# ------------------------------------------------------------------------------------------- residual step
LENS = [1, 70, 33, 130]
CUTS = {"whole": [[200]] * 4, "tokens": [[1]] * 4, "twos": [[2]] * 4,
        "mixed": [[1], [5, 1, 2, 40], [17, 16], [9, 64, 1, 2, 8, 7]]}


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("W,groups,K", [(96, 3, 4), (90, 1, 1), (90, 45, 2), (2048, 4, 4), (144, 6, 3), (264, 11, 6), (640, 2, 12),
                                        (4608, 9, 4), (2304, 1, 5), (63, 7, 0)])
def test_residual_step_with_norms_and_input_convolution(device, dtype, W, groups, K):
    """Two sublayers: the start from the embedding and a step behind a sublayer, in portions of every size."""
    eps, scale, V = 1e-5, 3.5, 50
    emb = rnd(V, W, seed=1, dtype=dtype)
    n1, n2, pw = (1 + rnd(W, seed=i, k=0.3) for i in (2, 3, 4))
    t1, t2 = rnd(max(K, 1), W, seed=5, k=0.5), rnd(max(K, 1), W, seed=6, k=0.5)
    ids = [torch.randint(0, V, (n,), generator=torch.Generator().manual_seed(n)).int() for n in LENS]
    ys = [rnd(n, W, seed=10 + n, dtype=dtype, k=4.0) for n in LENS]
    want = []
    for x, y in zip(ids, ys):
        e = d(emb)[x.long()] * scale
        h1 = oracle.group_norm(e, d(n1), groups, eps)
        x2 = e + oracle.group_norm(d(y), d(pw), groups, eps)
        h2 = oracle.group_norm(x2, d(n2), groups, eps)
        if K:
            h1, h2 = oracle.input_conv(h1, d(t1).T), oracle.input_conv(h2, d(t2).T)
        want.append((e, h1, x2, h2))
    dev = lambda t: t.to(device)                                            # noqa: E731
    for name, cuts in CUTS.items():
        hist = [torch.full((6, max(K - 1, 0), W), 9.0, device=device) for _ in range(2)]
        slots = [4, 1, 5, 2]
        for h in hist:
            h[slots] = 0.0
        got = [[[] for _ in range(4)] for _ in LENS]
        for step in portions(LENS, cuts):
            cu, sl = i32([0] + torch.tensor([c for _, _, c in step]).cumsum(0).tolist(), device), i32([slots[i] for i, _, _ in step], device)
            tok = dev(torch.cat([ids[i][a:a + c] for i, a, c in step]))
            y = dev(torch.cat([ys[i][a:a + c] for i, a, c in step]))
            ml = max(c for _, _, c in step)
            cv = lambda t, h: (dev(t), h, cu, sl, True) if K else None     # noqa: E731
            x1, h1 = ops.resid_start(dev(emb), tok, scale, dev(n1), groups, eps, cv(t1, hist[0]), max_len=ml)
            x2, h2 = ops.resid_step(x1, y, dev(pw), dev(n2), groups, eps, cv(t2, hist[1]), max_len=ml)
            at = 0
            for i, a, c in step:
                for k, t in enumerate((x1, h1, x2, h2)):
                    got[i][k].append(t[at:at + c])
                at += c
        for i in range(len(LENS)):
            for k, (g, w) in enumerate(zip(got[i], want[i])):
                close(torch.cat(g), w, torch.float32 if k in (0, 2) else dtype, 1e-5)
        for h in hist:
            assert bool((h[[0, 3]] == 9.0).all()), name                     # other slots are left alone


@pytest.mark.parametrize("device,dtype", WHERE)
def test_residual_step_without_writing_the_history(device, dtype):
    emb, taps, n1 = rnd(9, 64, seed=1, dtype=dtype, device=device), rnd(4, 64, seed=2, device=device), rnd(64, seed=3, device=device)
    hist = rnd(2, 3, 64, seed=4, device=device)
    keep = hist.clone()
    ops.resid_start(emb, i32([3, 4], device), 1.0, n1, 2, 1e-5, (taps, hist, i32([0, 2], device), i32([1], device), False), max_len=2)
    assert torch.equal(hist, keep)


# ------------------------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [
    (40, 3e5, 6.0, 2048, 24.0, 1.5), (20, 7e4, 8.0, 4096, 32.0, 1.0), (64, 1e4, 40.0, 4096, 32.0, 1.0), (2, 1e4, 2.0, 64, 8.0, 2.0),
    (8, 1e4, 1.0, 100, 32.0, 1.0), (24, 100.0, 3.0, 10, 32.0, 1.0), (24, 100.0, 3.0, 2, 32.0, 1.0), (12, 30.0, 0.5, 10 ** 7, 4.0, 2.0)])
def test_rotation_frequencies(dims, base, factor, original, fast, slow):
    """The table of a rotation with YaRN scaling, also where the ramp's ends meet or cross."""
    from legion_b200.models.decoder import Decoder
    dec = Decoder.__new__(Decoder)
    dec._rot, dec.device = {}, torch.device("cpu")
    tab = dec.rotary_table(RotarySpec(dims, base, factor, original, fast, slow), 300)
    rot = {"dims": dims, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    pos = torch.tensor([0, 1, 7, 63, 64, 150, 299])
    x = rnd(len(pos), 3, dims + 2, seed=1)
    want = oracle.rotate(x.double(), pos.tolist(), rot)
    assert torch.allclose(ops.reference.rotate_pairs(x, tab, pos).double(), want, atol=2e-6)
    f, m = oracle.frequencies(rot)
    assert torch.allclose(tab[299, :dims // 2].double(), torch.tensor([math.cos(299 * v) * m for v in f]).double(), atol=2e-6)


# ------------------------------------------------------------------------------------------- latent attention
def latent_case(H, dim, R, L, V, lens, qlens, page, device, dtype, loud=None, seed=0):
    """Latent rows of sequences in shuffled pages of a pool of large values, and the op's arguments for the sequences' last
    rows. ``loud`` = (sequence, position): its key answers one direction of every query, far above the others."""
    rot = {"dims": R, "base": 1e3, "scaling": {"factor": 2.0, "original": 100, "fast": 16.0, "slow": 1.0}}
    scale, eps = (dim + R) ** -0.5, 1e-5
    uk, uv = rnd(H * dim, L, seed=1, dtype=dtype, k=L ** -0.5), rnd(H * V, L, seed=2, dtype=dtype, k=L ** -0.5)
    nw = 1 + rnd(L, seed=3, k=0.2)
    from legion_b200.models.decoder import Decoder
    dec = Decoder.__new__(Decoder)
    dec._rot, dec.device = {}, torch.device(device)
    tab = dec.rotary_table(RotarySpec(R, 1e3, 2.0, 100, 16.0, 1.0), max(lens) + 1)
    row = -(-(L + R) // 8) * 8
    pages = [-(-n // page) for n in lens]
    order = torch.randperm(sum(pages) + 2, generator=torch.Generator().manual_seed(5)).tolist()
    cache = torch.full((len(order), page, 1, row), 50.0, dtype=dtype, device=device)
    bt = torch.zeros(len(lens), max(pages), dtype=torch.int32)
    for i, n in enumerate(pages):
        bt[i, :n] = torch.tensor([order.pop() for _ in range(n)])
    seqs = []
    for i, n in enumerate(lens):
        kv, q = rnd(n, L + R, seed=10 + i + seed, dtype=dtype), rnd(n, H, dim + R, seed=40 + i + seed, dtype=dtype)
        if loud is not None and loud[0] == i:
            p = loud[1]
            v = torch.sign(rnd(L, seed=77))                                 # the latent of the loud key, unlike all others
            kv[p, :L] = v.to(dtype)
            c = oracle.rms(v.double(), eps) * d(nw)
            for h in range(H):
                k = d(uk).view(H, dim, L)[h] @ c
                q[:, h, :dim] = (d(q[:, h, :dim]) * 0.05 + k / k.norm() ** 2 * 30.0 / scale).to(dtype)
            q[..., dim:] *= 0.05
        seqs.append((kv, q))
    return dict(rot=rot, scale=scale, eps=eps, uk=uk, uv=uv, nw=nw, tab=tab, cache=cache, bt=bt.to(device), seqs=seqs, page=page,
                H=H, dim=dim, R=R, L=L, V=V)


def latent_run(c, lens, qlens, gates, device, append_only=False):
    """The last qlens rows of every sequence through the ops, the rows before them appended in a first call."""
    H, dim, R, L = c["H"], c["dim"], c["R"], c["L"]
    slot = lambda i, p: int(c["bt"][i, p // c["page"]]) * c["page"] + p % c["page"]                     # noqa: E731
    uk_t = c["uk"].view(H, dim, L).transpose(1, 2).reshape(H * L, dim).contiguous().to(device)

    def feed(rows):
        kv = torch.cat([c["seqs"][i][0][a:b] for i, a, b in rows]).to(device)
        q = torch.cat([c["seqs"][i][1][a:b].reshape(b - a, -1) for i, a, b in rows]).to(device)
        pos = i32([p for _, a, b in rows for p in range(a, b)], device)
        slots = torch.tensor([slot(i, p) for i, a, b in rows for p in range(a, b)], dtype=torch.int64, device=device)
        return ops.latent_queries(q, kv, uk_t, c["nw"].to(device), c["eps"], c["tab"], pos, slots, c["cache"], H, dim, R)
    before = [(i, 0, n - m) for i, (n, m) in enumerate(zip(lens, qlens)) if n > m]
    if before:
        feed(before)
    if append_only:
        return None
    q_abs = feed([(i, n - m, n) for i, (n, m) in enumerate(zip(lens, qlens))])
    cu = i32([0] + torch.tensor(qlens).cumsum(0).tolist(), device)
    o = ops.latent_attention(q_abs, c["cache"], c["bt"], i32(lens, device), cu, max(qlens), c["scale"], L, R, max_ctx=max(lens))
    return ops.latent_values(o, c["uv"].to(device), None if gates is None else gates.to(device))


def latent_want(c, lens, qlens, gates):
    out, at = [], 0
    for (kv, q), n, m in zip(c["seqs"], lens, qlens):
        cl = oracle.rms(d(kv[:, :c["L"]]), c["eps"]) * d(c["nw"])
        kr = oracle.rotate(d(kv[:, c["L"]:]), range(n), c["rot"])
        qq = d(q[n - m:]).clone()
        qq[..., c["dim"]:] = oracle.rotate(qq[..., c["dim"]:], range(n - m, n), c["rot"])
        o = oracle.latent_heads(qq, cl, kr, d(c["uk"]), d(c["uv"]), c["scale"], c["dim"])
        if gates is not None:
            g = oracle.sigmoid(d(gates[at:at + m]))
            o = o * (g[:, :, None] if gates.shape[1] == c["H"] else g.view(o.shape))
        out.append(o.reshape(m, -1))
        at += m
    return torch.cat(out)


SIZES = [(4, 96, 32, 128, 80), (16, 128, 64, 512, 128), (3, 40, 24, 72, 32), (1, 13, 6, 19, 11), (6, 48, 16, 136, 40),
         (70, 16, 8, 64, 8), (5, 64, 64, 256, 96), (2, 32, 8, 320, 24), (128, 8, 16, 48, 16), (9, 24, 40, 504, 16)]


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,dim,R,L,V", SIZES)
@pytest.mark.parametrize("page", [64, 16])
def test_latent_attention_prompts_and_decode(device, dtype, H, dim, R, L, V, page):
    lens = [200, 64, 1, 131, 65]
    for n, qlens in enumerate(([70, 64, 1, 2, 1], [1] * 5, [200, 64, 1, 131, 65])):
        c = latent_case(H, dim, R, L, V, lens, qlens, page, device, dtype)
        T = sum(qlens)
        gates = [None, rnd(T, H, seed=9, dtype=dtype), rnd(T, H * V, seed=9, dtype=dtype)][(n + H) % 3]
        close(latent_run(c, lens, qlens, gates, device), latent_want(c, lens, qlens, gates), dtype, 2e-5, 1.5e-2)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("H,dim,R,L,V", [(4, 96, 32, 128, 80), (3, 128, 64, 512, 128), (3, 40, 24, 72, 32)])
def test_far_keys_at_page_and_split_borders(device, dtype, H, dim, R, L, V):
    """One key that outshines hundreds, at every border of pages and key splits: seen from prompts and from decode rows,
    and not seen by the rows in front of it."""
    n = 700
    for p in (0, 63, 64, 255, 256, n - 65, n - 2, n - 1):
        for m in (1, 90):
            c = latent_case(H, dim, R, L, V, [n, 30], [m, 1], 64, device, dtype, loud=(0, p))
            got, want = latent_run(c, [n, 30], [m, 1], None, device), latent_want(c, [n, 30], [m, 1], None)
            close(got, want, dtype, 2e-5, 2e-2)
            far = d(c["uv"]) @ (oracle.rms(d(c["seqs"][0][0][p, :L]), c["eps"]) * d(c["nw"]))
            for t in range(0, m, 13):                                       # the key decides every row that sees it
                off = float((want[t] - far).norm() / far.norm())
                assert off < 0.4 if p <= n - m + t else off > 0.6
    status_ok(device)


@gpu
@pytest.mark.parametrize("H,dim,R,L,V", [(4, 96, 32, 128, 80), (16, 128, 64, 512, 128), (3, 40, 24, 72, 32), (5, 64, 64, 256, 96),
                                         (2, 192, 64, 320, 256), (6, 48, 16, 136, 40)])
@pytest.mark.parametrize("page", [64, 16])
def test_fused_decode_and_per_head_prompts(H, dim, R, L, V, page):
    """The fused launches of decode steps, and steps whose long portions attend with keys and values per head beside short
    ones in the latent space; a loud key decides at page borders."""
    device, dtype = "cuda:0", torch.bfloat16
    bench = type("B", (), {})
    for lens, qlens in (([200, 64, 1, 131, 65], [1] * 5), ([700, 30], [1, 1]), ([300, 64, 700, 131, 1], [300, 64, 250, 1, 1]),
                        ([260], [200]), ([500, 193], [192, 193])):
        for loud in (None, (0, 63), (0, lens[0] - qlens[0])):
            c = latent_case(H, dim, R, L, V, lens, qlens, page, device, dtype, loud=loud)
            want = latent_want(c, lens, qlens, None)
            gates = [None, rnd(sum(qlens), H, seed=9, dtype=dtype), rnd(sum(qlens), H * V, seed=9, dtype=dtype)]
            latent_run(c, lens, qlens, None, device, append_only=True)
            q = torch.cat([x[1][n - m:].reshape(m, -1) for x, n, m in zip(c["seqs"], lens, qlens)]).to(device)
            kv = torch.cat([x[0][n - m:] for x, n, m in zip(c["seqs"], lens, qlens)]).to(device)
            uk_t = c["uk"].view(H, dim, L).transpose(1, 2).reshape(H * L, dim).contiguous().to(device)
            uk, uv, nw = c["uk"].to(device), c["uv"].to(device), c["nw"].to(device)
            host = [0] + torch.tensor(qlens).cumsum(0).tolist()
            b = bench()
            b.positions = i32([p for n, m in zip(lens, qlens) for p in range(n - m, n)], device)
            b.slots = torch.tensor([int(c["bt"][i, p // page]) * page + p % page for i, (n, m) in enumerate(zip(lens, qlens))
                                    for p in range(n - m, n)], device=device)
            b.cu_q, b.ctx_lens, b.block_table, b.token_ids = i32(host, device), i32(lens, device), c["bt"], b.positions
            b.n_seqs, b.max_q_len, b.max_ctx, b.cu_q_host, b.ctx_host, b.latent_parts = (len(lens), max(qlens), max(lens), host, lens,
                                                                                        None)
            for g in gates:
                gd = None if g is None else g.to(device)
                if max(qlens) == 1:
                    assert ops.sm100.latent_decode_ok(q, c["cache"], H, dim, R, L, V)
                    o = ops.sm100.latent_decode(q, kv, gd, uk_t, uv, nw, c["eps"], c["tab"], b.positions, b.slots, c["cache"],
                                                b.block_table, b.ctx_lens, b.cu_q, c["scale"], H, dim, R, max(lens))
                else:
                    o = torch.zeros(sum(qlens), H * V, dtype=dtype, device=device)
                    parts = ops.sm100.latent_parts(b, page)
                    assert [p.expand for p in parts] == ([True, False] if min(qlens) < 192 else [True])
                    for p in parts:
                        sel = (lambda t: t) if p.rows is None else (lambda t: t.index_select(0, p.rows))      # noqa: E731
                        qp, kvp, gp = sel(q), sel(kv), None if gd is None else sel(gd)
                        if p.expand:
                            assert ops.sm100.latent_expand_ok(qp, c["cache"], p, H, dim, R, R, L, V)
                            r = ops.sm100.latent_prompt(qp, kvp, gp, uk, uv, nw, c["eps"], c["tab"], c["cache"], p, c["scale"], H, dim, R)
                        else:
                            qa = ops.latent_queries(qp, kvp, uk_t, nw, c["eps"], c["tab"], p.positions, p.slots, c["cache"], H, dim, R)
                            r = ops.latent_values(ops.latent_attention(qa, c["cache"], p.block_table, p.ctx_lens, p.cu_q, p.max_q_len,
                                                                       c["scale"], L, R, max_ctx=p.max_ctx), uv, gp)
                        o = r if p.rows is None else o.index_copy_(0, p.rows, r)
                x = want
                if g is not None:
                    s = oracle.sigmoid(d(g))
                    x = (want.view(-1, H, V) * (s[:, :, None] if g.shape[1] == H else s.view(-1, H, V))).reshape(want.shape)
                close(o, x, dtype, 2e-5, 2e-2)
    status_ok(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_padding_rows_leave_the_cache_alone(device, dtype):
    c = latent_case(4, 96, 32, 128, 80, [70], [1], 64, device, dtype)
    before = c["cache"].clone()
    q, kv = c["seqs"][0][1].reshape(70, -1)[:2].to(device), c["seqs"][0][0][:2].to(device)
    ops.latent_queries(q, kv, rnd(4 * 128, 96, dtype=dtype, device=device), c["nw"].to(device), 1e-5, c["tab"], i32([0, 0], device),
                       torch.tensor([-1, -1], device=device), c["cache"], 4, 96, 32)
    assert torch.equal(before, c["cache"])


# ------------------------------------------------------------------------------------------- gated recurrence
def lru_weights(W, blocks, K, dtype):
    dd = W // blocks
    return dict(in_b=rnd(W, seed=1, k=0.3), conv_w=rnd(W, K, seed=2, k=0.5), conv_b=rnd(W, seed=3, k=0.2),
                ra=rnd(blocks, dd, dd, seed=4, dtype=dtype, k=1.5 * dd ** -0.5), ri=rnd(blocks, dd, dd, seed=5, dtype=dtype, k=1.5 * dd ** -0.5),
                ra_b=rnd(blocks, dd, seed=6, k=0.5), ri_b=rnd(blocks, dd, seed=7, k=0.5),
                lam=torch.log(torch.expm1(0.001 + 0.3 * torch.rand(W, generator=torch.Generator().manual_seed(8)) ** 3)), y_b=rnd(W, seed=9, k=0.3))


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("W,blocks,K", [(96, 3, 4), (640, 5, 4), (21, 1, 1), (35, 35, 3), (512, 1, 2), (90, 2, 9), (256, 2, 4), (512, 2, 4),
                                        (192, 3, 7)])
def test_gated_recurrence_prompts_portions_and_decode(device, dtype, W, blocks, K):
    """Convolution, gates, recurrence and GELU branch; every portion size, states of other slots untouched."""
    w, dd = lru_weights(W, blocks, K, dtype), W // blocks
    lens = [1, 70, 33, 200]
    xs, ys = [rnd(n, W, seed=20 + n, dtype=dtype) for n in lens], [rnd(n, W, seed=60 + n, dtype=dtype) for n in lens]
    want = []
    for x, y in zip(xs, ys):
        u = oracle.short_conv(d(x) + d(w["in_b"]), d(w["conv_w"]), d(w["conv_b"]))
        if dtype == torch.bfloat16:
            u = u.bfloat16().double()
        r = oracle.sigmoid(oracle.block_product(u, d(w["ra"]), d(w["ra_b"])))
        i = oracle.sigmoid(oracle.block_product(u, d(w["ri"]), d(w["ri_b"])))
        S, last = oracle.gated_recurrence(u, r, i, d(w["lam"]))
        want.append((S * oracle.gelu_tanh(d(y) + d(w["y_b"])), last))
    g = {k: v.to(device) for k, v in w.items()}
    gw = torch.stack([g["ra"], g["ri"]], 1).reshape(-1, dd).contiguous()
    gb = torch.stack([g["ra_b"], g["ri_b"]], 1).reshape(-1).contiguous()
    ld = (-8 * torch.nn.functional.softplus(g["lam"].double())).float()
    for name, cuts in CUTS.items():
        conv, state = torch.full((6, W, K - 1), 9.0, device=device), torch.full((6, W), 9.0, device=device)
        slots = [4, 1, 5, 2]
        conv[slots], state[slots] = 0.0, 0.0
        got = [[] for _ in lens]
        for step in portions(lens, cuts):
            host = [0] + torch.tensor([c for _, _, c in step]).cumsum(0).tolist()
            cu, sl = i32(host, device), i32([slots[i] for i, _, _ in step], device)
            # column slices of one projection, as in the model
            xy = torch.cat([torch.cat([ys[i][a:a + c], xs[i][a:a + c]], 1) for i, a, c in step]).to(device)
            y, x = xy[:, :W], xy[:, W:]
            ml = max(c for _, _, c in step)
            if device != "cpu" and ml == 1:
                o = ops.sm100.rglru_decode(x, g["in_b"], g["conv_w"], g["conv_b"], conv, gw, gb, ld, y, g["y_b"], state, cu, sl, blocks)
            else:
                u = ops.causal_conv1d_silu(x, g["conv_w"], g["conv_b"], conv, cu, sl, max_len=ml, in_bias=g["in_b"], silu=False)
                o = ops.gated_recurrence(u, ops.block_gates(u, gw, blocks), gb, ld, y, g["y_b"], state, cu, sl, blocks, max_len=ml,
                                         cu_host=host)
            for (i, _, c), a in zip(step, host):
                got[i].append(o[a:a + c])
        for i in range(len(lens)):
            close(torch.cat(got[i]), want[i][0], dtype, 2e-5, 1.5e-2)
            close(state[slots[i]], want[i][1], dtype, 2e-5, 1.5e-2)
        assert bool((state[[0, 3]] == 9.0).all()) and bool((conv[[0, 3]] == 9.0).all()), name
    status_ok(device)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,blocks,n", [(2560, 10, 64), (1280, 5, 70), (640, 20, 9), (256, 1, 17), (96, 1, 33)])
def test_gated_recurrence_decode_of_many_sequences(dtype, W, blocks, n):
    """One token of each of n sequences from random histories and states, in slots in no order."""
    device, K = "cuda:0", 4
    w, dd = lru_weights(W, blocks, K, dtype), W // blocks
    conv, state = rnd(n + 3, W, K - 1, seed=31), rnd(n + 3, W, seed=32)
    x, y = rnd(n, W, seed=33, dtype=dtype), rnd(n, W, seed=34, dtype=dtype)
    slots = torch.randperm(n + 3, generator=torch.Generator().manual_seed(35))[:n]
    win = torch.cat([d(conv)[slots], (d(x) + d(w["in_b"]))[:, :, None]], 2)
    u = (win * d(w["conv_w"])).sum(2) + d(w["conv_b"])
    u = u.bfloat16().double() if dtype == torch.bfloat16 else u
    r, i = (oracle.sigmoid(oracle.block_product(u, d(w[k]), d(w[k + "_b"]))) for k in ("ra", "ri"))
    S = torch.stack([oracle.gated_recurrence(u[j:j + 1], r[j:j + 1], i[j:j + 1], d(w["lam"]), d(state)[slots[j]])[1] for j in range(n)])
    g = {k: v.to(device) for k, v in w.items()}
    gw = torch.stack([g["ra"], g["ri"]], 1).reshape(-1, dd).contiguous()
    gb = torch.stack([g["ra_b"], g["ri_b"]], 1).reshape(-1).contiguous()
    ld = (-8 * torch.nn.functional.softplus(g["lam"].double())).float()
    cv, st = conv.to(device), state.to(device)
    o = ops.sm100.rglru_decode(x.to(device), g["in_b"], g["conv_w"], g["conv_b"], cv, gw, gb, ld, y.to(device), g["y_b"], st,
                               i32(list(range(n + 1)), device), slots.int().to(device), blocks)
    close(o, S * oracle.gelu_tanh(d(y) + d(w["y_b"])), dtype, 2e-5, 1.5e-2)
    close(st[slots.to(device)], S, dtype, 2e-5, 1.5e-2)
    close(cv[slots.to(device)], win[:, :, 1:], torch.float32, 1e-6)
    rest = [j for j in range(n + 3) if j not in set(slots.tolist())]
    assert torch.equal(st[rest].cpu(), state[rest]) and torch.equal(cv[rest].cpu(), conv[rest])


@pytest.mark.parametrize("device,dtype", WHERE)
def test_recurrence_keeps_a_slow_state(device, dtype):
    """Decays near one over hundreds of tokens: an early input is still there, across chunk edges."""
    W, n = 64, 500
    u, y = torch.zeros(n, W, dtype=dtype), torch.full((n, W), 3.0, dtype=dtype)
    u[0] = 1.0
    gates = torch.zeros(n, 2 * W)
    ld = torch.full((W,), -2e-3)
    b = torch.cat([torch.full((W,), 1.0), torch.full((W,), -1.0)])
    S, _ = oracle.gated_recurrence(d(u), oracle.sigmoid(torch.full((n, W), 1.0).double()), oracle.sigmoid(torch.full((n, W), -1.0).double()),
                                   torch.log(torch.expm1(-d(ld) / 8)))
    state = torch.zeros(1, W, device=device)
    o = ops.gated_recurrence(u.to(device), gates.to(device), b.to(device), ld.to(device), y.to(device), torch.zeros(W, device=device),
                             state, i32([0, n], device), i32([0], device), 1, max_len=n, cu_host=[0, n])
    close(o, S * oracle.gelu_tanh(d(y)), dtype, 1e-4)
    assert float(o[-1].float().abs().min()) > 0.1 * float(o[0].float().abs().min())


# ------------------------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,K,N", [(1, 64, 96), (5, 2048, 512), (300, 256, 200), (33, 90, 27), (64, 4096, 128), (7, 72, 1030)])
@pytest.mark.parametrize("p,q", [(0.3, -0.8), (-2.0, 1.5)])
def test_xielu_in_the_projection(device, dtype, T, K, N, p, q):
    x, w = rnd(T, K, seed=1, dtype=dtype), rnd(N, K, seed=2, dtype=dtype, k=2 * K ** -0.5)
    pq = torch.tensor([p, q]).double()
    ab = (oracle.softplus(pq) + torch.tensor([0.0, 0.5]).double()).float().to(device)
    got = ops.up_act(x.to(device), w.to(device), ab)
    close(got, oracle.xielu(d(x) @ d(w).T, pq[0], pq[1]), dtype)
    status_ok(device)
