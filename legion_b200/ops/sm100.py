"""Python front-ends of the sm_100a kernels in ``legion_b200/_C.so``.

Every function takes CUDA tensors, enqueues on the current stream and never synchronises; scratch
(split-K partials, attention split buffers, routing plans) comes from a per-device ``Workspace`` that
is allocated once, so a decode step captured in a CUDA graph replays without allocator traffic.
The extension is required on a GPU: there is no silent fallback to eager PyTorch.
"""
from __future__ import annotations

import importlib
import os
import threading
from typing import Optional

import torch

_C = None
_C_err: Optional[BaseException] = None
_lock = threading.Lock()


# kernels launched by one call of each binding (for the launch counter)
KERNELS_PER_CALL = {"moe_plan": 3, "paged_decode": 1, "argmax": 2, "wgemm_workspace_floats": 0, "linear_chunk": 3, "linear_chunk_ok": 0, "tmap_encoded": 0,
                    "linear_chunk_scratch_bytes": 0, "conv_silu_any": 2}
LAUNCHES = {"n": 0}


class _Counting:
    """Proxy of the extension module that counts kernel launches (``LAUNCHES['n']``) and, with ``LB_OP_PROFILE=1``
    (or ``op_profile(True)``), times every op between two CUDA events: the per-op table of the reference's
    ``LEGION_OP_PROFILE`` (``src/ggml/op_profile.rs:1-16``). Profiling is for eager steps (run with
    ``--no-cuda-graphs``); captured graphs replay without passing through here."""

    def __init__(self, mod):
        self._mod = mod
        self._cache = {}

    def __getattr__(self, name):
        f = self._cache.get(name)
        if f is None:
            raw = getattr(self._mod, name)
            k = KERNELS_PER_CALL.get(name, 1)

            def f(*a, _raw=raw, _k=k, _name=name, **kw):
                LAUNCHES["n"] += _k
                if not OP_PROFILE["on"] or _k == 0 or torch.cuda.is_current_stream_capturing():
                    return _raw(*a, **kw)
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                out = _raw(*a, **kw)
                e1.record()
                OP_PROFILE["events"].append((_name, e0, e1))
                return out
            self._cache[name] = f
        return f


OP_PROFILE = {"on": os.environ.get("LB_OP_PROFILE", "0") == "1", "events": []}


def op_profile(on: bool):
    OP_PROFILE["on"] = bool(on)
    OP_PROFILE["events"].clear()


def op_profile_report(reset: bool = True):
    """Rows (op, calls, total ms, mean us, share) of the ops timed since the last report, slowest first."""
    torch.cuda.synchronize()
    agg = {}
    for name, e0, e1 in OP_PROFILE["events"]:
        c = agg.setdefault(name, [0, 0.0])
        c[0] += 1
        c[1] += e0.elapsed_time(e1)
    if reset:
        OP_PROFILE["events"].clear()
    total = sum(v[1] for v in agg.values()) or 1.0
    return [(n, c, ms, ms / c * 1e3, ms / total) for n, (c, ms) in sorted(agg.items(), key=lambda kv: -kv[1][1])]


def ext():
    """Returns the extension module, importing ``legion_b200._C`` on first use."""
    global _C, _C_err
    if _C is None and _C_err is None:
        with _lock:
            if _C is None and _C_err is None:
                try:
                    mod = _import_ext()
                    mod.set_pdl(bool(TUNE["pdl"]))
                    _C = _Counting(mod)
                except BaseException as e:  # missing .so, ABI mismatch, missing libcudart
                    _C_err = e
    if _C is None:
        raise RuntimeError(
            "legion_b200._C (the sm_100a extension) is not importable: build it with "
            "`python -m legion_b200.build_ext`") from _C_err
    return _C


def _import_ext():
    """The full extension ``_C``, or the subset ``_C_core`` in a checkout where only that one was built (its absent kernels
    stay unresolved)."""
    import sys
    from importlib.util import find_spec
    name = "legion_b200._C"
    if find_spec(name) is None and find_spec("legion_b200._C_core") is not None:
        flags = sys.getdlopenflags()
        sys.setdlopenflags(os.RTLD_LAZY)
        try:
            return importlib.import_module("legion_b200._C_core")
        finally:
            sys.setdlopenflags(flags)
    return importlib.import_module(name)


def have_ext() -> bool:
    try:
        ext()
        return True
    except RuntimeError:
        return False


NUM_SMS = 148

# tuning knobs (environment: LB_TUNE="decode_fixed_tiles=2,dense_route=1")
TUNE = {"parallel_branches": 3, "decode_lanes": 2, "nv4_sorted": 1, "fp8_fused_quant": 1, "nv4_sorted_bn": 64, "gdn_chunk": 1, "decode_fixed_tiles": 2, "fused_plan": 1, "fused_router": 1, "dense_route": 1, "pdl": 1, "route_norm": 0, "mla_head_gemm": 1}
for _kv in os.environ.get("LB_TUNE", "").split(","):
    if "=" in _kv:
        TUNE[_kv.split("=")[0].strip()] = int(_kv.split("=")[1])


_CANARY_ON = os.environ.get("LB_CANARY", "0") == "1"


class Workspace:
    """Per-device scratch shared by all kernels on that device's compute stream. A decode step that runs as several
    concurrent lanes (``engine.cuda_graphs``: independent halves of the batch on parallel branches of one CUDA graph)
    gives every lane a workspace of its own: ``Workspace.lane`` selects it while that lane's launches are issued."""

    _by_device: dict = {}
    lane: int = 0

    def __init__(self, device: torch.device):
        self.device = device
        self.status = torch.zeros(4, dtype=torch.int32, device=device)
        self.counters = torch.zeros(1 << 16, dtype=torch.int32, device=device)
        self.splitk = torch.empty(1 << 23, dtype=torch.float32, device=device)  # 32 MiB
        self._attn: dict = {}
        self._cache: dict = {}
        self._guards: dict = {}

    @classmethod
    def get(cls, device) -> "Workspace":
        device = torch.device(device)
        if device.index is None:
            device = torch.device("cuda", torch.cuda.current_device())
        key = device if cls.lane == 0 else (device, cls.lane)
        ws = cls._by_device.get(key)
        if ws is None:
            ws = cls(device)
            cls._by_device[key] = ws
        return ws

    CANARY_BYTES = 256
    CANARY = 0xA5

    def buf(self, key, shape, dtype):
        """A cached scratch tensor: same key and size -> same storage (graph-safe). With ``LB_CANARY=1`` every buffer
        sits between two guard areas filled with a byte pattern that ``check_canaries`` verifies: the substitute
        for a memory checker on kernels that index scratch memory (a write past either end shows up by name)."""
        k = (key, tuple(shape), dtype)
        t = self._cache.get(k)
        if t is None:
            if _CANARY_ON:
                n = 1
                for d in shape:
                    n *= int(d)
                nbytes = n * torch.empty(0, dtype=dtype).element_size()
                pad = self.CANARY_BYTES
                raw = torch.full((nbytes + 2 * pad,), self.CANARY, dtype=torch.uint8, device=self.device)
                t = raw[pad:pad + nbytes].view(dtype).view(shape)
                self._guards[k] = raw
            else:
                t = torch.empty(shape, dtype=dtype, device=self.device)
            self._cache[k] = t
        return t

    def check_canaries(self) -> list:
        """Names of the scratch buffers whose guard areas no longer hold the pattern (``LB_CANARY=1`` only)."""
        bad = []
        pad = self.CANARY_BYTES
        for k, raw in self._guards.items():
            if bool((raw[:pad] != self.CANARY).any()) or bool((raw[-pad:] != self.CANARY).any()):
                bad.append(str(k[0]))
        return bad

    def check(self) -> int:
        """Synchronises and returns the kernels' status word (0 = ok); clears it."""
        v = int(self.status[0].item())
        if v:
            self.status.zero_()
        for key, other in list(self._by_device.items()):      # the other lanes of this device
            if isinstance(key, tuple) and key[0] == self.device and other is not self:
                ov = int(other.status[0].item())
                if ov:
                    other.status.zero_()
                    v = v or ov
        return v


class QWeight:
    """NVFP4 weight kept in its 4-bit encoding: ``codes`` uint8 [..., rows, K/2] (two e2m1 values per byte, low
    nibble first), ``scales`` uint8 e4m3 bit patterns [..., rows, K/16], ``gscale`` float32 per tensor (per expert;
    for a fused gate/up tensor two values per expert: gate, up). The GEMM streams the 4-bit bytes and expands
    them to bf16 operand tiles inside the kernel (``csrc/gemm_sm100.cu``), so a decode step reads 0.56 bytes per
    weight instead of 2."""
    __slots__ = ("codes", "scales", "gscale")

    def __init__(self, codes, scales, gscale):
        self.codes, self.scales, self.gscale = codes, scales.view(torch.uint8), gscale.float().reshape(-1).contiguous()

    @property
    def shape(self):
        return tuple(self.codes.shape[:-1]) + (self.codes.shape[-1] * 2,)

    @property
    def device(self):
        return self.codes.device

    def dim(self):
        return self.codes.dim()

    def view2d(self):
        return self.codes.reshape(-1, self.codes.shape[-1]), self.scales.reshape(-1, self.scales.shape[-1])

    def narrow(self, lo: int, hi: int) -> "QWeight":
        """Groups [lo, hi) of a stacked weight (a view: no copy). hi == lo + 1 with ``squeeze`` semantics is
        ``narrow(lo, lo + 1).squeeze0()``."""
        per = self.gscale.numel() // self.codes.shape[0]
        return QWeight(self.codes[lo:hi], self.scales[lo:hi], self.gscale[lo * per:hi * per])

    def squeeze0(self) -> "QWeight":
        return QWeight(self.codes[0], self.scales[0], self.gscale)

    @classmethod
    def quantize(cls, w: torch.Tensor, dual_rows: int = 0):
        """Encodes a bf16/fp32 weight [..., rows, K] (tests, synthetic checkpoints). ``dual_rows`` > 0: the tensor is
        a fused [gate | up] stack of 2 * dual_rows rows and each half gets its own tensor scale."""
        from ..loaders.quant_formats import nvfp4_quant
        lead = w.shape[:-2]
        flat = w.reshape(-1, w.shape[-2], w.shape[-1])
        codes, scales, gs = [], [], []
        for t in flat:
            parts = [t] if not dual_rows else [t[:dual_rows], t[dual_rows:]]
            cs, ss = [], []
            for part in parts:
                c, sc, g = nvfp4_quant(part.float().cpu())
                cs.append(c)
                ss.append(sc.view(torch.uint8))
                gs.append(float(g))
            codes.append(torch.cat(cs, 0))
            scales.append(torch.cat(ss, 0))
        dev = w.device
        return cls(torch.stack(codes).reshape(*lead, *codes[0].shape).to(dev),
                   torch.stack(scales).reshape(*lead, *scales[0].shape).to(dev),
                   torch.tensor(gs, dtype=torch.float32, device=dev))

    @classmethod
    def quantize_cuda(cls, w: torch.Tensor, dual_rows: int = 0):
        """Device-side encoding of a CUDA bf16 weight [..., rows, K] (``csrc/quant.cu::nvfp4_quant``): one tensor
        scale per leading index (two with ``dual_rows``: gate rows, up rows)."""
        C = ext()
        rows, K = w.shape[-2], w.shape[-1]
        flat = w.reshape(-1, rows, K)
        n = flat.shape[0]
        codes = torch.empty(n, rows, K // 2, dtype=torch.uint8, device=w.device)
        scales = torch.empty(n, rows, K // 16, dtype=torch.uint8, device=w.device)
        per = 2 if dual_rows else 1
        gs = torch.empty(n * per, dtype=torch.float32, device=w.device)
        for t in range(n):
            for h in range(per):
                r0, r1 = (0, rows) if not dual_rows else (h * dual_rows, (h + 1) * dual_rows)
                part = flat[t, r0:r1]
                g = (part.float().abs().max() / (6.0 * 448.0)).clamp_min(1e-12).reshape(1)
                gs[t * per + h] = g[0]
                C.nvfp4_quant(part.contiguous(), g, codes[t, r0:r1], scales[t, r0:r1])
        lead = tuple(w.shape[:-2])
        return cls(codes.reshape(*lead, rows, K // 2), scales.reshape(*lead, rows, K // 16), gs)

    def dequantize(self, dtype=torch.bfloat16):
        from ..loaders.quant_formats import nvfp4_dequant
        c2, s2 = self.view2d()
        rows = self.codes.shape[-2]
        n_t = c2.shape[0] // rows
        per = self.gscale.numel() // n_t
        out = torch.empty(c2.shape[0], c2.shape[1] * 2, dtype=dtype, device=self.device)
        for t in range(n_t):
            for h in range(per):
                r0 = t * rows + h * (rows // per)
                r1 = r0 + rows // per
                out[r0:r1] = nvfp4_dequant(c2[r0:r1].cpu(), s2[r0:r1].cpu(), float(self.gscale[t * per + h]),
                                           out_dtype=dtype).to(self.device)
        return out.reshape(self.shape)


class Nv4Weight:
    """NVFP4 weight in the layout of the native block-scaled GEMM (``csrc/gemm_nvfp4_sm100.cu``): ``codes`` uint8
    [..., rows, K/2] exactly as shipped (two e2m1 values per byte, low nibble first), ``sf`` the UE4M3 block scales
    re-ordered into 512-byte atoms (128 rows x 4 blocks, the order tcgen05.cp wants; same bytes, other order),
    ``gscale`` float32 per tensor (per expert; two per expert for a fused gate/up stack). Rows per leading index
    must be a multiple of 128. Activations are quantised to NVFP4 as well (W4A4), so the tensor cores run the
    e2m1 x e2m1 block-scaled instruction and nothing is expanded."""
    __slots__ = ("codes", "sf", "gscale", "scales_lin")

    def __init__(self, codes, sf, gscale, scales_lin=None):
        self.codes, self.sf, self.gscale = codes, sf, gscale.float().reshape(-1).contiguous()
        self.scales_lin = scales_lin          # kept only when asked for (tests / de-quantisation)

    @property
    def shape(self):
        return tuple(self.codes.shape[:-1]) + (self.codes.shape[-1] * 2,)

    @property
    def device(self):
        return self.codes.device

    def dim(self):
        return self.codes.dim()

    def view2d(self):
        return self.codes.reshape(-1, self.codes.shape[-1])

    @classmethod
    def from_parts(cls, codes, scales, gscale, keep_linear: bool = False):
        """From the checkpoint tensors: codes [..., rows, K/2], scales e4m3 bytes [..., rows, K/16], tensor scale(s)."""
        C = ext()
        rows = codes.shape[-2]
        if codes.dim() > 2 and rows % 128:
            raise ValueError("stacked NVFP4 weights need a multiple of 128 rows per slice")
        c2 = codes.reshape(-1, codes.shape[-1]).contiguous()
        s2 = scales.view(torch.uint8).reshape(-1, scales.shape[-1]).contiguous()
        K = c2.shape[1] * 2
        atoms = torch.zeros(C.nv4_sf_bytes(c2.shape[0], K), dtype=torch.uint8, device=codes.device)
        C.nv4_pack_scales(s2, atoms)
        return cls(codes.contiguous(), atoms, gscale, s2 if keep_linear else None)

    @classmethod
    def from_qweight(cls, q: "QWeight", keep_linear: bool = False):
        return cls.from_parts(q.codes, q.scales, q.gscale, keep_linear)

    @classmethod
    def quantize_cuda(cls, w: torch.Tensor, dual_rows: int = 0, keep_linear: bool = False):
        return cls.from_qweight(QWeight.quantize_cuda(w, dual_rows), keep_linear)

    def narrow(self, lo: int, hi: int) -> "Nv4Weight":
        """Groups [lo, hi) of a stacked weight (views of the same storage)."""
        n, rows = self.codes.shape[0], self.codes.shape[-2]
        per = self.gscale.numel() // n
        bpg = self.sf.numel() // n                    # scale-atom bytes per group (rows are a multiple of 128)
        lin = None
        if self.scales_lin is not None:
            lin = self.scales_lin[lo * rows:hi * rows]
        return Nv4Weight(self.codes[lo:hi], self.sf[lo * bpg:hi * bpg], self.gscale[lo * per:hi * per], lin)

    def squeeze0(self) -> "Nv4Weight":
        return Nv4Weight(self.codes[0], self.sf, self.gscale, self.scales_lin)

    def as_qweight(self) -> "QWeight":
        """The same weight with its block scales in the checkpoint's linear order (for the de-quantising GEMM that
        serves prompt-sized steps); the linear copy is made on first use and kept."""
        if self.scales_lin is None:
            C = ext()
            c2 = self.view2d()
            K = c2.shape[1] * 2
            lin = torch.empty(c2.shape[0], K // 16, dtype=torch.uint8, device=self.device)
            C.nv4_unpack_scales(self.sf, lin)
            self.scales_lin = lin
        K16 = self.codes.shape[-1] // 8
        return QWeight(self.codes, self.scales_lin.view(*self.codes.shape[:-1], K16), self.gscale)

    def dequantize(self, dtype=torch.bfloat16):
        return self.as_qweight().dequantize(dtype)


class Nv4Act:
    """NVFP4-encoded activation rows: codes [T, K/2], scale atoms, and the fp32 scale (one per row, or one device
    scalar for all rows when ``stride`` is 0)."""
    __slots__ = ("codes", "sf", "gscale", "stride", "normed", "summed")

    def __init__(self, codes, sf, gscale, stride, normed=None, summed=None):
        self.codes, self.sf, self.gscale, self.stride, self.normed, self.summed = codes, sf, gscale, stride, normed, summed

    def dequantize(self):
        C = ext()
        T, K = self.codes.shape[0], self.codes.shape[1] * 2
        lin = torch.empty(T, K // 16, dtype=torch.uint8, device=self.codes.device)
        C.nv4_unpack_scales(self.sf, lin)
        from ..loaders.quant_formats import nvfp4_dequant
        out = nvfp4_dequant(self.codes.cpu(), lin.cpu(), 1.0, out_dtype=torch.float32).to(self.codes.device)
        g = self.gscale.reshape(-1)[:1] if self.stride == 0 else self.gscale[:T]
        return out * g.reshape(-1, 1)


def nv4_quant_act(x, norm=None, residual=None, static_scale=None, want_normed: bool = False, key=None):
    """bf16 rows [T, K] -> ``Nv4Act``. ``norm=(weight, eps, w_offset)`` fuses the RMSNorm that produces the rows
    (and ``residual`` the add before it: ``summed`` is then the new residual stream); ``static_scale`` is a device
    scalar used for every row instead of the per-row amax scale. ``key``: reuse the same output storage on every
    call with that key (graph-safe)."""
    C = ext()
    T, K = x.shape
    ws = Workspace.get(x.device)
    if key is not None:
        codes = ws.buf((key, "c"), (T, K // 2), torch.uint8)
        sf = ws.buf((key, "s"), (C.nv4_sf_bytes(T, K),), torch.uint8)
        gs = ws.buf((key, "g"), (max(T, 1),), torch.float32) if static_scale is None else static_scale
    else:
        codes = torch.empty(T, K // 2, dtype=torch.uint8, device=x.device)
        sf = torch.empty(C.nv4_sf_bytes(T, K), dtype=torch.uint8, device=x.device)
        gs = torch.empty(max(T, 1), dtype=torch.float32, device=x.device) if static_scale is None else static_scale
    normed = torch.empty_like(x) if (want_normed and norm is not None) else None
    summed = torch.empty_like(x) if residual is not None else None
    C.nv4_act_quant(x, residual, summed, norm[0] if norm else None, norm[1] if norm else 0.0, norm[2] if norm else 0.0,
                    normed, static_scale, codes, sf, None if static_scale is not None else gs)
    return Nv4Act(codes, sf, gs, 0 if static_scale is not None else 1, normed, summed)


def linear_nv4(xq: "Nv4Act", w: "Nv4Weight", residual=None, out=None, bn=None):
    """out[T, N] = dequant(xq) @ dequant(w)^T (+ residual) on the native NVFP4 tensor-core path."""
    C = ext()
    T = xq.codes.shape[0]
    N = w.shape[0]
    if out is None:
        out = torch.empty(T, N, dtype=torch.bfloat16, device=xq.codes.device)
    if T == 0:
        return out
    ws = Workspace.get(xq.codes.device)
    bn = bn or (32 if T <= 32 else (64 if T <= 64 else 128))
    C.wgemm_nv4(w.view2d(), w.sf, w.gscale, xq.codes, xq.sf, xq.gscale, xq.stride, out, residual, None, None, N, False,
                0, 0, bn, ws.status, None, None, None, None, 0, 0, T, None, None, None, None)
    return out


def gate_up_nv4(xq: "Nv4Act", w: "Nv4Weight", n_ff: int, act: str = "silu", out=None, q_scale=None, bn=None):
    """act(x Wg^T) * (x Wu^T) with Wg = w[:n_ff], Wu = w[n_ff:]. With ``q_scale`` (device scalar) the result is
    returned NVFP4-encoded (``Nv4Act`` with that static tensor scale) for the next GEMM."""
    C = ext()
    T = xq.codes.shape[0]
    dev = xq.codes.device
    ws = Workspace.get(dev)
    bn = bn or (32 if T <= 32 else 64)
    a = 0 if act == "silu" else 1
    if q_scale is not None:
        qc = torch.empty(T, n_ff // 2, dtype=torch.uint8, device=dev)
        qs = torch.zeros(C.nv4_sf_bytes(T, n_ff), dtype=torch.uint8, device=dev)
        C.wgemm_nv4(w.view2d(), w.sf, w.gscale, xq.codes, xq.sf, xq.gscale, xq.stride, None, None, None, None, n_ff,
                    True, n_ff, a, bn, ws.status, None, None, None, None, 0, 0, T, None, qc, qs, q_scale)
        return Nv4Act(qc, qs, q_scale, 0)
    if out is None:
        out = torch.empty(T, n_ff, dtype=torch.bfloat16, device=dev)
    C.wgemm_nv4(w.view2d(), w.sf, w.gscale, xq.codes, xq.sf, xq.gscale, xq.stride, out, None, None, None, n_ff, True,
                n_ff, a, bn, ws.status, None, None, None, None, 0, 0, T, None, None, None, None)
    return out


def pick_bn(n_tok: int, dual: bool) -> int:
    bn = 32
    cap = 128 if dual else 256
    while bn < n_tok and bn < cap:
        bn *= 2
    return bn


def _pick_split_k(n_tok_tiles: int, feat_tiles: int, K: int) -> int:
    """Split K when a skinny GEMM has too few tiles to keep the SMs streaming weights."""
    tiles = n_tok_tiles * feat_tiles
    num_kb = (K + 63) // 64
    if tiles >= NUM_SMS // 2 or num_kb < 8:
        return 1
    s = min(NUM_SMS // max(tiles, 1), num_kb // 4, 16)
    return max(1, s)


class Fp8Weight:
    """Block-scaled FP8 weight kept in its 8-bit encoding: ``data`` uint8 e4m3 bit patterns [..., rows, K] and
    ``scale`` float32 per 128 x 128 block [..., ceil(rows / 128), K / 128] (the layout of FP8 checkpoints with
    ``weight_block_size = [128, 128]``; ``weight_scale_inv`` is this scale). The GEMM feeds the bytes straight to
    the e4m3 tensor-core instruction, with the activations quantised per token and 128 columns, and adds each
    128-wide k block with its two scales in fp32 (``csrc/gemm_sm100.cu``, FP8 mode): a decode step reads one byte
    per weight instead of two."""
    __slots__ = ("data", "scale")

    def __init__(self, data, scale):
        self.data, self.scale = data.view(torch.uint8), scale.float().contiguous()

    @property
    def shape(self):
        return tuple(self.data.shape)

    @property
    def device(self):
        return self.data.device

    def dim(self):
        return self.data.dim()

    def view2d(self):
        return self.data.reshape(-1, self.data.shape[-1]), self.scale.reshape(-1, self.scale.shape[-1])

    def narrow(self, lo: int, hi: int) -> "Fp8Weight":
        return Fp8Weight(self.data[lo:hi], self.scale[lo:hi])

    def squeeze0(self) -> "Fp8Weight":
        return Fp8Weight(self.data[0], self.scale[0])

    @classmethod
    def quantize(cls, w: torch.Tensor):
        """Device-side encoding of a CUDA bf16 weight [..., rows, K] (rows a multiple of 128 when stacked)."""
        C = ext()
        rows, K = w.shape[-2], w.shape[-1]
        if K % 128 or (w.dim() > 2 and rows % 128):
            raise ValueError("FP8 block scaling needs K % 128 == 0 and 128-row aligned stacks")
        flat = w.reshape(-1, K).contiguous()
        data = torch.empty(flat.shape, dtype=torch.uint8, device=w.device)
        scale = torch.empty((flat.shape[0] + 127) // 128, K // 128, dtype=torch.float32, device=w.device)
        C.fp8_block_quant(flat, 128, 128, data, scale)
        lead = tuple(w.shape[:-2])
        return cls(data.view(*lead, rows, K), scale.view(*lead, (rows + 127) // 128, K // 128) if lead else scale)

    def dequantize(self, dtype=torch.bfloat16):
        C = ext()
        d2, s2 = self.view2d()
        out = torch.empty(d2.shape, dtype=torch.bfloat16, device=d2.device)
        C.fp8_block_dequant(d2.contiguous(), s2.contiguous(), 128, 128, out)
        return out.view(self.shape).to(dtype)


class Fp8Act:
    """Activation rows already encoded for the FP8 GEMMs (e4m3 bytes + one scale per row and 128 columns), kept with
    the bf16 rows they came from: a layer input that feeds several FP8 projections is encoded once."""
    __slots__ = ("x", "data", "scale")

    def __init__(self, x, data, scale):
        self.x, self.data, self.scale = x, data, scale

    is_cuda = True

    @property
    def shape(self):
        return self.x.shape

    @property
    def device(self):
        return self.x.device

    @classmethod
    def of(cls, x):
        d, s = fp8_quant_act(x)
        return cls(x, d, s)


def _fp8_parts(x):
    return (x.data, x.scale) if isinstance(x, Fp8Act) else fp8_quant_act(x)


def fp8_quant_act(x, out=None, scale=None):
    """bf16 activations [T, K] -> (e4m3 bytes [T, K], fp32 scale per row and 128 columns [T, K / 128])."""
    C = ext()
    T, K = x.shape
    if out is None:
        out = torch.empty(T, K, dtype=torch.uint8, device=x.device)
        scale = torch.empty(T, K // 128, dtype=torch.float32, device=x.device)
    C.fp8_act_quant(x, out, scale)
    return out, scale


def _linear_fp8(x, w: "Fp8Weight", residual, out, dual: bool, n_feat: int):
    C = ext()
    T, K = x.shape
    ws = Workspace.get(x.device)
    x8, xs = _fp8_parts(x)
    bn = 32 if T <= 32 else 64
    n_tt = (T + bn - 1) // bn
    ft = (n_feat + 127) // 128
    sk = _pick_split_k(n_tt, ft, K)
    if sk > 1:
        need = C.wgemm_workspace_floats(bn, dual, n_tt, ft, sk)
        if need > ws.splitk.numel() or n_tt * ft > ws.counters.numel():
            sk = 1
    w2, s2 = w.view2d()
    C.wgemm_fp8(w2, s2, x8, xs, out, residual, None, None, n_feat, dual, n_feat if dual else 0, bn, sk,
                ws.splitk if sk > 1 else None, ws.counters if sk > 1 else None, ws.status, None, None, None, None, 0, 0,
                T, None)
    return out


ROUTER_MODES = {"softmax": 0, "sigmoid": 1, "softmax_bias": 2, "biased_softmax": 3}
RENORM = {False: 0, True: 1, "sum": 2}       # see config.MoeSpec.renorm
GATE_ACTS = {"silu": 0, "gelu_tanh": 1, "relu2": 2}


def tma_ok(*ts) -> bool:
    """bf16 operands whose rows TMA can fetch (16-byte aligned base and row pitch)."""
    return all(t.dtype == torch.bfloat16 and t.shape[-1] % 8 == 0 and t.stride(-2) % 8 == 0 and t.data_ptr() % 16 == 0
               for t in ts)


def sgemm(x, w, residual=None, out=None, out_dtype=None, dual: bool = False, n_ff: int = 0, act: str = "silu",
          act_ab=None, unary: Optional[str] = None, tok_scale=None, bias=None):
    """x @ w^T in fp32 arithmetic on the FMA units: fp32 models and shapes outside the tcgen05 GEMM's alignment rules.
    ``dual``: act(x Wg^T) * (x Wu^T) with Wg = w[:n_ff], Wu = w[n_ff:]."""
    T, N = x.shape[0], (n_ff if dual else w.shape[0])
    if out is None:
        out = torch.empty(T, N, dtype=out_dtype or x.dtype, device=x.device)
    ext().sgemm(w, x, out, residual, tok_scale, None, N, dual, n_ff if dual else 0,
                3 if act_ab is not None else GATE_ACTS[unary] if unary else GATE_ACTS[act] if dual else 0, None, None, None, None, 0, 0, T, act_ab, bias)
    return out


def up_act(x, w, ab):
    """xIELU(x @ w^T) with the activation in the epilogue; ``ab``: its two numbers, float32."""
    return linear(x, w, out_dtype=x.dtype, xielu=ab)


def linear(x, w, residual=None, out=None, out_dtype=torch.bfloat16, split_k: Optional[int] = None, bn=None, xielu=None,
           unary: Optional[str] = None, tok_scale=None):
    """out[T, N] = x[T, K] @ w[N, K]^T (+ residual). ``unary``: "relu2"; ``tok_scale`` (float32): a factor per row."""
    C = ext()
    if isinstance(w, torch.Tensor) and isinstance(x, torch.Tensor) and not tma_ok(x, w):
        return sgemm(x, w, residual, out, out_dtype, act_ab=xielu, unary=unary, tok_scale=tok_scale)
    if (xielu is not None or unary is not None or tok_scale is not None) and not isinstance(w, torch.Tensor):
        raise ValueError("activations and row factors run in the epilogue of bf16 and fp32 weights")
    if isinstance(x, Fp8Act) and not isinstance(w, Fp8Weight):
        x = x.x
    T, K = x.shape
    N = w.shape[0]
    q = isinstance(w, QWeight)
    if q and out_dtype != torch.bfloat16:
        raise ValueError("NVFP4 weights produce bf16 outputs")
    if out is None:
        out = torch.empty(T, N, dtype=out_dtype, device=x.device)
    if T == 0:
        return out
    if isinstance(w, Fp8Weight):
        if out_dtype != torch.bfloat16:
            raise ValueError("FP8 weights produce bf16 outputs")
        return _linear_fp8(x, w, residual, out, False, N)
    if isinstance(w, Nv4Weight):
        if out_dtype != torch.bfloat16:
            raise ValueError("NVFP4 weights produce bf16 outputs")
        return linear_nv4(x if isinstance(x, Nv4Act) else nv4_quant_act(x), w, residual=residual, out=out)
    ws = Workspace.get(x.device)
    bn = bn or pick_bn(T, False)
    n_tt = (T + bn - 1) // bn
    ft = (N + 127) // 128
    sk = _pick_split_k(n_tt, ft, K) if split_k is None else split_k
    if sk > 1:
        need = C.wgemm_workspace_floats(bn, False, n_tt, ft, sk)
        if need > ws.splitk.numel() or n_tt * ft > ws.counters.numel():
            sk = 1
    C.wgemm(w.codes if q else w, x, out, residual, tok_scale, None, N, False, 0, bn, sk, ws.splitk if sk > 1 else None,
            ws.counters if sk > 1 else None, ws.status, None, None, None, None, 0, 0, T, [], None,
            w.scales if q else None, w.gscale if q else None, xielu=xielu, relu2=unary == "relu2")
    return out


def gate_up_act(x, w_gate_up, n_ff: int, out=None, bn=None, split_k: Optional[int] = None, act: str = "silu", bias=None):
    """act(x @ Wg^T) * (x @ Wu^T) with Wg = w_gate_up[:n_ff], Wu = w_gate_up[n_ff:] (GELU and ``bias``, float32 [bg | bu] added
    ahead of the activation: bf16 and fp32 weights only)."""
    C = ext()
    if isinstance(w_gate_up, torch.Tensor) and isinstance(x, torch.Tensor) and not tma_ok(x, w_gate_up):
        return sgemm(x, w_gate_up, None, out, None, True, n_ff, act, bias=bias)
    if bias is not None and not isinstance(w_gate_up, torch.Tensor):
        raise ValueError("biases run in the epilogue of bf16 and fp32 weights")
    if isinstance(x, Fp8Act) and not isinstance(w_gate_up, Fp8Weight):
        x = x.x
    T, K = x.shape
    if out is None:
        out = torch.empty(T, n_ff, dtype=torch.bfloat16, device=x.device)
    if T == 0:
        return out
    if isinstance(w_gate_up, Fp8Weight):
        return _linear_fp8(x, w_gate_up, None, out, True, n_ff)
    if isinstance(w_gate_up, Nv4Weight):
        return gate_up_nv4(x if isinstance(x, Nv4Act) else nv4_quant_act(x), w_gate_up, n_ff, out=out)
    ws = Workspace.get(x.device)
    bn = bn or pick_bn(T, True)
    n_tt = (T + bn - 1) // bn
    ft = (n_ff + 127) // 128
    sk = _pick_split_k(n_tt, ft, K) if split_k is None else split_k
    if sk > 1:
        need = C.wgemm_workspace_floats(bn, True, n_tt, ft, sk)
        if need > ws.splitk.numel() or n_tt * ft > ws.counters.numel():
            sk = 1
    q = isinstance(w_gate_up, QWeight)
    C.wgemm(w_gate_up.codes if q else w_gate_up, x, out, None, None, None, n_ff, True, n_ff, bn, sk,
            ws.splitk if sk > 1 else None, ws.counters if sk > 1 else None, ws.status, None, None, None, None, 0, 0, T,
            [], None, w_gate_up.scales if q else None, w_gate_up.gscale if q else None, 0, 0, GATE_ACTS[act], bias=bias)
    return out


def rmsnorm(x, w, eps, w_offset=0.0, residual=None, out=None, sum_out=None):
    """Returns (normed, summed). With a residual the sum x + residual is the new residual stream."""
    C = ext()
    if out is None:
        out = torch.empty_like(x)
    if residual is not None and sum_out is None:
        sum_out = torch.empty_like(x)
    C.rmsnorm(x, residual, sum_out, w, out, eps, w_offset)
    return out, (sum_out if residual is not None else x)


def qk_norm_rope_append(qkv, n_q, n_kv, d, q_norm_w, k_norm_w, eps, w_offset, cos_sin, rot, positions, slots,
                        k_cache, v_cache, gated_q=False, q_out=None):
    C = ext()
    T = qkv.shape[0]
    if q_out is None:
        q_out = torch.empty(T, n_q, d, dtype=torch.bfloat16, device=qkv.device)
    qhs = 2 * d if gated_q else d
    k_off = n_q * qhs
    v_off = k_off + n_kv * d
    C.qk_norm_rope_append(qkv, qhs, k_off, v_off, q_norm_w, k_norm_w, eps, w_offset, cos_sin, rot, positions, slots,
                          q_out, k_cache, v_cache, n_q, n_kv, d)
    return q_out


def sigmoid_gate(attn, qkv, n_q, d, out=None):
    C = ext()
    if out is None:
        out = torch.empty_like(attn)
    C.sigmoid_gate(attn, qkv, 2 * d, d, n_q, out)
    return out


def decode_splits(batch: int, n_kv_heads: int, g_tiles: int, max_ctx: int, head_dim: int = 128) -> int:
    """Flash-decoding split count. The grid is (batch x kv heads x head tiles x splits) CTAs, one resident per SM
    (its K/V rings take most of the shared memory), and a split covers ceil(tiles / splits) 128-key tiles. The
    count minimises waves x (tiles per split + fixed cost per CTA): 2.2 waves cost as much as 3, and a count
    that leaves the last split empty only adds idle CTAs."""
    ctas = max(1, batch * n_kv_heads * g_tiles)
    slots = NUM_SMS
    tiles = max(1, (max_ctx + 127) // 128)
    fixed = TUNE["decode_fixed_tiles"]
    best, best_cost = 1, None
    for s in range(1, min(128, tiles) + 1):
        per = (tiles + s - 1) // s
        if (tiles + per - 1) // per != s:
            continue
        waves = (ctas * s + slots - 1) // slots
        cost = waves * (per + fixed)
        if best_cost is None or cost < best_cost:
            best, best_cost = s, cost
    return best


def paged_decode(q, k_cache, v_cache, block_table, ctx_lens, scale, window=0, n_splits=None, max_ctx=None, out=None,
                 impl="tc", softcap=0.0):
    C = ext()
    B, Hq, _ = q.shape
    Hkv, D = k_cache.shape[2], v_cache.shape[3]
    if n_splits is None:
        G = Hq // Hkv
        span = max_ctx or block_table.shape[1] * k_cache.shape[1]
        if window > 0:
            span = min(span, window + 128)            # tiles a window can touch
        n_splits = decode_splits(B, Hkv, (G + 15) // 16, span, D)
    ws = Workspace.get(q.device)
    o_part = ws.buf("dec_o", (B * Hq * n_splits * 2 * D,), torch.float32)
    ml_part = ws.buf("dec_ml", (B * Hq * n_splits * 2 * 2,), torch.float32)
    if out is None:
        out = torch.empty(B, Hq, D, dtype=q.dtype, device=q.device)
    C.paged_decode(q, k_cache, v_cache, block_table, ctx_lens, scale, window, n_splits, o_part, ml_part, out,
                   impl == "tc", ws.status, ws.counters, float(softcap))
    return out


def prefill_attn(q, k_cache, v_cache, cu_q, ctx_lens, block_table, max_q_len, scale, window=0, causal=True, out=None,
                 softcap=0.0):
    C = ext()
    if out is None:
        out = torch.empty(q.shape[0], q.shape[1], v_cache.shape[3], dtype=q.dtype, device=q.device)
    ws = Workspace.get(q.device)
    C.prefill_attn(q, k_cache, v_cache, cu_q, ctx_lens, block_table, max_q_len, scale, window, causal, out, ws.status,
                   float(softcap))
    return out


def attention_ext(q, k_cache, v_cache, block_table, ctx_lens, cu_q, max_q_len, scale, window=0, keep_first=0, sink=None, gate=None,
                  out_scale=1.0, out=None, n_splits=None, max_ctx=None):
    """Paged causal attention with sinks, first tokens that stay visible behind the window, a gate per head, an output scale
    and output rows that may lie apart ([T, heads * value head size])."""
    C = ext()
    T, Hq, _ = q.shape
    Hkv, D = k_cache.shape[2], v_cache.shape[3]
    if out is None:
        out = torch.empty(T, Hq * D, dtype=q.dtype, device=q.device)
    if T == 0:
        return out
    aligned = out.data_ptr() % 16 == 0 and out.stride(0) % 8 == 0
    if not (attn_tc_ok(q, k_cache, v_cache) and aligned):
        C.paged_attn_general(q, k_cache, v_cache, cu_q, ctx_lens, block_table, scale, window, out, 0.0, keep_first, sink, gate,
                             out_scale)
        return out
    ws = Workspace.get(q.device)
    if max_q_len > 1:
        C.prefill_attn_ext(q, k_cache, v_cache, cu_q, ctx_lens, block_table, max_q_len, scale, window, out, ws.status, keep_first,
                           sink, gate, out_scale)
        return out
    if n_splits is None:
        span = max_ctx or block_table.shape[1] * k_cache.shape[1]
        if window > 0:
            span = min(span, window + 128 + -(-keep_first // 128) * 128)       # tiles that can hold visible tokens
        n_splits = decode_splits(T, Hkv, (Hq // Hkv + 15) // 16, span, D)
    o_part = ws.buf("dec_o", (T * Hq * n_splits * 2 * D,), torch.float32)
    ml_part = ws.buf("dec_ml", (T * Hq * n_splits * 2 * 2,), torch.float32)
    C.paged_decode_ext(q, k_cache, v_cache, block_table, ctx_lens, scale, window, n_splits, o_part, ml_part, out, ws.status,
                       ws.counters, keep_first, sink, gate, out_scale)
    return out


def attn_tc_ok(q, k_cache, v_cache) -> bool:
    """Whether the tcgen05 attention kernels take these caches: bf16, head sizes that are multiples of 8 up to 256."""
    dk, dv, page = k_cache.shape[3], v_cache.shape[3], k_cache.shape[1]
    return (q.dtype == torch.bfloat16 and dk % 8 == 0 and dv % 8 == 0 and dk <= 256 and dv <= 256 and page % 8 == 0
            and 64 % page == 0)


def paged_attn_general(q, k_cache, v_cache, block_table, ctx_lens, cu_q, scale, window=0, causal=True, out=None, softcap=0.0):
    """Paged causal attention for fp32 and for head sizes outside the tensor-core kernels (prompts and decode rows)."""
    if not causal:
        raise NotImplementedError("the general attention kernel is causal")
    if out is None:
        out = torch.empty(q.shape[0], q.shape[1], v_cache.shape[3], dtype=q.dtype, device=q.device)
    ext().paged_attn_general(q, k_cache, v_cache, cu_q, ctx_lens, block_table, scale, window, out, float(softcap))
    return out


def qkv_norm_append(q, k, v, q_norm, k_norm, eps, slots, k_cache, v_cache):
    """q, k, v: column slices of one projection. Head norms (plain weights, optional), k and v to their cache cells;
    returns the queries [T, heads, dk]. Any head sizes, bf16 or fp32."""
    q_out = torch.empty(q.shape[0], q.shape[1] // k_cache.shape[3], k_cache.shape[3], dtype=q.dtype, device=q.device)
    ext().qkv_norm_append(q, k, v, q_norm, k_norm, eps, slots, q_out, k_cache, v_cache)
    return q_out


def head_linear(x, w2d, n_heads: int, rows_per_group: int, n_feat: int, K: int, x_group_col: int, out2d):
    """Per-head projections read and written in place: for every head h
    ``out2d[t * n_heads + h, :n_feat] = W_h @ x[t, h * x_group_col : h * x_group_col + K]`` (0: every head reads the
    same K columns) with
    ``W_h = w2d[h * rows_per_group : h * rows_per_group + n_feat]``. One grouped launch of the tcgen05 GEMM (group =
    head); the activation tile of a head is fetched from its column slice of ``x`` by the TMA load, the output rows
    go through a row map, so nothing is transposed or copied."""
    C = ext()
    T = x.shape[0]
    if not (tma_ok(x, w2d) and x_group_col % 8 == 0):
        # fp32 and unaligned shapes: the FMA kernel
        C.sgemm_heads(w2d, x, out2d.view(T, -1), n_heads, rows_per_group, n_feat, K, x_group_col, out2d.shape[1])
        return out2d
    ws = Workspace.get(x.device)
    bn = pick_bn(T, False)
    key = ("head_linear", T, n_heads, bn)
    tab = ws._cache.get(key)
    if tab is None:
        n_tt = (T + bn - 1) // bn
        Tp = n_tt * bn
        h = torch.arange(n_heads).repeat_interleave(n_tt)
        tt = torch.arange(n_tt).repeat(n_heads)
        rows = torch.full((n_heads * Tp,), -1, dtype=torch.int32)
        t = torch.arange(T)
        for hh in range(n_heads):
            rows[hh * Tp: hh * Tp + T] = (t * n_heads + hh).int()
        i32 = dict(dtype=torch.int32, device=x.device)
        tab = (h.to(**i32), (tt * bn).to(**i32), torch.clamp(T - tt * bn, max=bn).to(**i32),
               (h * Tp + tt * bn).to(**i32), rows.to(x.device),
               torch.tensor([n_heads * n_tt, 0], **i32), n_heads * n_tt)
        ws._cache[key] = tab
    tile_group, tile_tok0, tile_ntok, tile_out0, out_rows, meta, n_tiles = tab
    C.wgemm(w2d, x, out2d, None, None, out_rows, n_feat, False, 0, bn, 1, None, None, ws.status, tile_group, tile_tok0,
            tile_ntok, meta, n_tiles, rows_per_group, 0, [], tile_out0, None, None, x_group_col, K if x_group_col else 0)
    return out2d


def mla_splits(n_seqs: int, max_q_len: int, nh: int, max_ctx: int) -> int:
    """Key splits of the latent-attention kernel: enough CTAs (64 query rows each) to cover the SMs, at least four
    64-key tiles per split."""
    g = min(nh, 64)
    tiles = max(1, n_seqs * ((max_q_len + 64 // g - 1) // (64 // g)) * max(1, nh // 64))
    by_sm = max(1, NUM_SMS // tiles)
    by_len = max(1, (max_ctx + 255) // 256)
    return int(max(1, min(by_sm, by_len, 32)))


def mla_supported(nh: int, kv_lora: int, rope_dim: int, page: int) -> bool:
    return kv_lora == 512 and rope_dim == 64 and page % 8 == 0 and 64 % page == 0 and \
        ((nh >= 64 and nh % 64 == 0) or (0 < nh < 64 and 64 % nh == 0))


def mla_prep(kva, norm_w, eps, w_offset, q, q_pe_off, cos_sin, positions, slots, cache, q_abs):
    """Cache row [rmsnorm(c_kv) | rope(k_pe)] written at each token's cell and rope(q_pe) written into
    q_abs[..., 512:] in one launch."""
    ext().mla_prep(kva, norm_w, eps, w_offset, q, q_pe_off, cos_sin, positions, slots, cache, q_abs)


def mla_attn(q_abs, cache, cu_q, ctx_lens, block_table, page, max_q_len, scale, n_splits=None, max_ctx=None, out=None,
             rank: int = 512, rot: int = 64):
    """Latent attention, absorbed form: q_abs [T, heads, rank + rot], cache rows [.., rank + rot] (either with padding
    columns behind) -> [T, heads, rank]."""
    C = ext()
    T, nh, _ = q_abs.shape
    if n_splits is None:
        n_splits = mla_splits(int(ctx_lens.numel()), max_q_len, nh, max_ctx or block_table.shape[1] * page)
    ws = Workspace.get(q_abs.device)
    o_part = ml_part = None
    if n_splits > 1:
        o_part = ws.buf("mla_o", (T * nh * n_splits * rank,), torch.float32)
        ml_part = ws.buf("mla_ml", (T * nh * n_splits * 2,), torch.float32)
    if out is None:
        out = torch.empty(T, nh, rank, dtype=torch.bfloat16, device=q_abs.device)
    C.mla_attn(q_abs, cache, cu_q, ctx_lens, block_table, page, max_q_len, scale, n_splits, o_part, ml_part, out, rank, rot,
               True, ws.status)
    return out


def latent_tc_ok(q_abs, cache, rank: int, rot: int) -> bool:
    """Whether the tcgen05 latent-attention kernel takes these rows."""
    page = cache.shape[1]
    return (q_abs.dtype == torch.bfloat16 and rank % 8 == 0 and (rank + rot) % 8 == 0 and rank <= 512 and rank + rot <= 576
            and q_abs.shape[2] % 8 == 0 and cache.shape[-1] % 8 == 0 and page % 8 == 0 and 64 % page == 0)


def latent_row(rank: int, rot: int) -> int:
    """Columns of a query row in the latent space, padded so that rows start on 16-byte boundaries."""
    return -(-(rank + rot) // 8) * 8


def latent_queries(q, kv, uk, norm_w, eps, cos_sin, positions, slots, cache, heads: int, dim: int, rot_dim: int):
    """Cache rows of the step's tokens and the queries in the latent space, [T, heads, rank + rot_dim] (rows padded to
    multiples of 8 columns)."""
    T, L = q.shape[0], norm_w.numel()
    q_abs = torch.empty(T, heads, latent_row(L, rot_dim), dtype=q.dtype, device=q.device)
    head_linear(q, uk, heads, L, L, dim, dim + rot_dim, q_abs.view(T * heads, -1))
    ext().latent_prep(q, kv, norm_w, eps, cos_sin, positions, slots, cache, q_abs, dim, rot_dim, None, False)
    return q_abs


LATENT_DECODE_ROWS = 64      # most rows of a step on the fused decode launches


def latent_decode_ok(q, cache, heads: int, dim: int, rot: int, rank: int, vdim: int) -> bool:
    """Whether a decode step runs on the fused launches around the tcgen05 latent attention."""
    page = cache.shape[1]
    return (q.dtype == torch.bfloat16 and q.shape[0] <= LATENT_DECODE_ROWS and rank % 8 == 0 and (rank + rot) % 8 == 0
            and rank <= 512 and rank + rot <= 576 and dim % 4 == 0 and dim <= 256 and (dim + rot) % 4 == 0
            and q.stride(0) % 4 == 0 and q.data_ptr() % 8 == 0 and page % 8 == 0 and 64 % page == 0)


def latent_decode(q, kv, gate, uk, uv, norm_w, eps, cos_sin, positions, slots, cache, block_table, ctx_lens, cu_q, scale,
                  heads: int, dim: int, rot: int, max_ctx=None):
    """One token per sequence: queries into the latent space with the cache append | attention over the latents in key
    splits | merge, value projection and output gate. [T, heads * vdim]."""
    C = ext()
    T, L, page = q.shape[0], norm_w.numel(), cache.shape[1]
    ws = Workspace.get(q.device)
    bf = dict(dtype=torch.bfloat16, device=q.device)
    q_abs = torch.empty(T, heads, latent_row(L, rot), **bf)
    C.latent_prep(q, kv, norm_w, eps, cos_sin, positions, slots, cache, q_abs, dim, rot, uk, False)
    n = mla_splits(int(ctx_lens.numel()), 1, heads, max_ctx or block_table.shape[1] * page)
    o_part = ml_part = o_lat = None
    if n > 1:
        o_part = ws.buf("mla_o", (T * heads * n * L,), torch.float32)
        ml_part = ws.buf("mla_ml", (T * heads * n * 2,), torch.float32)
    else:
        o_lat = torch.empty(T, heads, L, **bf)
    C.mla_attn(q_abs, cache, cu_q, ctx_lens, block_table, page, 1, scale, n, o_part, ml_part, o_lat, L, rot, False, ws.status)
    out = torch.empty(T, uv.shape[0], **bf)
    C.latent_decode_v(o_part, ml_part, n, o_lat, uv, gate, heads, L, out)
    return out


LATENT_EXPAND_MIN = 192      # portions from this many tokens attend in the per-head form
LATENT_EXPAND_BYTES = 2 << 30    # ... while the expanded keys and values stay below this


class LatentPart:
    """Sequences of a step that run in one form of latent attention. ``rows``: their rows in the step (None: all of it)."""
    __slots__ = ("expand", "rows", "positions", "slots", "cu_q", "ctx_lens", "block_table", "max_q_len", "max_ctx", "pages",
                 "table")


def latent_parts(b, page: int) -> list:
    """Splits a step's sequences into long portions (per-head form) and the rest (latent space); kept with the batch for
    its other layers. Without host copies of the lengths everything runs in the latent space."""
    if b.latent_parts is not None:
        return b.latent_parts
    cu, ctx, dev = b.cu_q_host, b.ctx_host, b.token_ids.device
    lens = [cu[i + 1] - cu[i] for i in range(len(cu) - 1)] if cu is not None else []
    long = [i for i, n in enumerate(lens) if n >= LATENT_EXPAND_MIN] if ctx is not None else []
    rest = [i for i, n in enumerate(lens) if i not in set(long) and n > 0]

    def part(seqs, expand):
        p = LatentPart()
        p.expand, p.pages, p.table = expand, None, None
        if len(seqs) == b.n_seqs:
            p.rows, p.positions, p.slots, p.cu_q, p.ctx_lens, p.block_table = (None, b.positions, b.slots, b.cu_q, b.ctx_lens,
                                                                               b.block_table)
            p.max_q_len, p.max_ctx = b.max_q_len, b.max_ctx
        else:
            p.rows = torch.tensor([r for i in seqs for r in range(cu[i], cu[i + 1])], dtype=torch.int64, device=dev)
            at = [0]
            for i in seqs:
                at.append(at[-1] + lens[i])
            sel = torch.tensor(seqs, dtype=torch.int64, device=dev)
            p.positions, p.slots = b.positions.index_select(0, p.rows), b.slots.index_select(0, p.rows)
            p.cu_q = torch.tensor(at, dtype=torch.int32, device=dev)
            p.ctx_lens, p.block_table = b.ctx_lens.index_select(0, sel), b.block_table.index_select(0, sel)
            p.max_q_len = max(lens[i] for i in seqs)
            p.max_ctx = max(ctx[i] for i in seqs) if ctx is not None else b.max_ctx
        if expand:
            n = [-(-ctx[i] // 64) for i in seqs]
            p.pages = torch.tensor([[j for j, k in enumerate(n) for _ in range(k)], [64 * x for k in n for x in range(k)]],
                                   dtype=torch.int32, device=dev)
            t, first = torch.zeros(len(seqs), max(n), dtype=torch.int32), 0
            for j, k in enumerate(n):
                t[j, :k] = torch.arange(first, first + k)
                first += k
            p.table = t.to(dev)
        return p
    if not long:
        p = part(list(range(b.n_seqs)), False)
        parts = [p]
    else:
        parts = [part(long, True)] + ([part(rest, False)] if rest else [])
    b.latent_parts = parts
    return parts


def latent_expand_ok(q, cache, p: LatentPart, heads: int, dim: int, rot: int, rot_cols: int, rank: int, vdim: int) -> bool:
    return (p.expand and q.dtype == torch.bfloat16 and dim % 8 == 0 and rot % 8 == 0 and rot_cols == rot and rank % 8 == 0
            and vdim % 8 == 0 and dim + rot <= 256 and vdim <= 256 and cache.shape[-1] % 8 == 0 and q.stride(0) % 8 == 0
            and q.data_ptr() % 16 == 0 and p.pages.shape[1] * 64 * heads * (dim + rot + vdim) * 2 <= LATENT_EXPAND_BYTES)


def latent_prompt(q, kv, gate, uk_rows, uv, norm_w, eps, cos_sin, cache, p: LatentPart, scale, heads: int, dim: int, rot: int):
    """Long portions: the sequences' cached latents become keys and values of every head (one product each), attended by
    the prefill kernel. Per visible pair that is dim + rot + vdim products instead of 2 rank + rot in the latent space.
    ``uk_rows`` [heads * dim, rank]. [T, heads * vdim]."""
    C = ext()
    T, L, n = q.shape[0], norm_w.numel(), p.pages.shape[1]
    V = uv.shape[0] // heads
    bf = dict(dtype=torch.bfloat16, device=q.device)
    qf = torch.empty(T, heads, dim + rot, **bf)
    C.latent_prep(q, kv, norm_w, eps, cos_sin, p.positions, p.slots, cache, qf, dim, rot, None, True)
    lat, k = torch.empty(n * 64, L, **bf), torch.empty(n * 64, heads, dim + rot, **bf)
    C.latent_gather(cache, p.block_table, p.ctx_lens, p.pages, lat, k, dim, rot)
    head_linear(lat, uk_rows, heads, dim, dim, L, 0, k.view(n * 64 * heads, dim + rot))
    v = linear(lat, uv)
    o = prefill_attn(qf, k.view(n, 64, heads, dim + rot), v.view(n, 64, heads, V), p.cu_q, p.ctx_lens, p.table, p.max_q_len,
                     scale).view(T, heads * V)
    if gate is not None:
        C.latent_gate(o, gate, heads)
    return o


def latent_attention(q_abs, cache, block_table, ctx_lens, cu_q, max_q_len, scale, rank: int, rot: int, max_ctx=None):
    """Causal attention over cached latent rows, [T, heads, rank]: tcgen05 in bf16, FMA units for fp32 and other sizes."""
    if latent_tc_ok(q_abs, cache, rank, rot):
        return mla_attn(q_abs, cache, cu_q, ctx_lens, block_table, cache.shape[1], max_q_len, scale, max_ctx=max_ctx, rank=rank,
                        rot=rot)
    out = torch.empty(q_abs.shape[0], q_abs.shape[1], rank, dtype=q_abs.dtype, device=q_abs.device)
    ext().latent_attn_general(q_abs, cache, cu_q, ctx_lens, block_table, scale, rank, rot, out)
    return out


def latent_values(o_lat, uv, gate):
    """Per-head value projection of the attended latents and the output gate: [T, heads * vdim]."""
    T, H, L = o_lat.shape
    vdim = uv.shape[0] // H
    out = torch.empty(T, H * vdim, dtype=o_lat.dtype, device=o_lat.device)
    head_linear(o_lat.view(T, H * L), uv, H, vdim, vdim, L, L, out.view(T * H, vdim))
    if gate is not None:
        ext().latent_gate(out, gate, H)
    return out


def router_topk(logits, k, mode="softmax", renorm=True, route_scale=1.0, bias=None, n_group=1, topk_group=1,
                ids=None, wts=None, group_top: int = 2, gate=None):
    """``gate`` (float32 [T]) takes the sigmoid of the logits' last column, which then is no expert."""
    C = ext()
    T = logits.shape[0]
    if ids is None:
        ids = torch.empty(T, k, dtype=torch.int32, device=logits.device)
        wts = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    C.router_topk(logits, bias, k, ROUTER_MODES[mode], RENORM[renorm], route_scale, n_group, topk_group, ids, wts, group_top,
                  gate)
    return ids, wts


class Routing:
    """Router result of one step: ``ids`` / ``wts`` [T, k] and, for decode-sized steps, the dense routing tables
    (``dense``) that let the expert GEMMs run without a gather. Unpacks as ``ids, wts = routing``."""
    __slots__ = ("ids", "wts", "dense", "x_normed", "e_lo", "n_local", "shared_slot", "xq", "gate", "shared_rows")

    def __init__(self, ids, wts, dense=None, x_normed=None, e_lo=0, n_local=None):
        self.ids, self.wts, self.dense, self.x_normed = ids, wts, dense, x_normed
        self.e_lo, self.n_local = e_lo, n_local      # expert range the dense tables were built for
        self.shared_slot = False                     # the shared expert has a slot of its own in the dense tables
        self.xq = None                               # the experts' input already NVFP4-encoded (Nv4Act)
        self.gate = None                             # [T] sigmoid gate of a shared expert that runs by itself
        self.shared_rows = 0                         # always-chosen experts in the dense tables, behind a token's pairs

    def __iter__(self):
        yield self.ids
        yield self.wts


class DenseRoute:
    """Device tables of the dense routing (one token tile per active expert covering all T tokens). ``bn`` is the
    token tile of the GEMMs, ``stride`` the distance between the rows of consecutive slots in the intermediate
    tensor (= bn, or 128 for the NVFP4 path whose 32-token tiles must start a 128-row scale atom), ``n_slots`` the
    most slots a step can have (local experts, + 1 when the shared expert is stacked behind them)."""

    def __init__(self, n_slots: int, bn: int, device, stride: Optional[int] = None):
        i32 = dict(dtype=torch.int32, device=device)
        self.n_slots, self.bn, self.stride = n_slots, bn, stride or bn
        self.E = n_slots
        self.tile_group = torch.zeros(n_slots, **i32)
        self.slot_base = torch.zeros(n_slots, **i32)
        self.zeros = torch.zeros(n_slots, **i32)
        self.tile_ntok = torch.zeros(n_slots, **i32)
        self.meta = torch.zeros(2, **i32)
        self.out_rows = torch.full((n_slots * self.stride,), -1, **i32)
        self.tok_scale = torch.zeros(n_slots * self.stride, dtype=torch.float32, device=device)
        self.h8 = self.h8_scale = None               # FP8 experts: the activated rows, encoded by the gate/up GEMM
        self.sh_logit = torch.zeros(4 * 64, dtype=torch.float32, device=device)   # one plane per column split
        self.active = torch.zeros(n_slots, **i32)      # per local expert: chosen by some token of the step
        self.h_all = None
        self.hq = None
        self.y_pairs = None


def router(x, w_router, k, mode="softmax", renorm=True, route_scale=1.0, bias=None, n_group=1, topk_group=1,
           norm=None, e_lo: int = 0, n_local: Optional[int] = None, slot_stride: Optional[int] = None, sh_gate=None,
           shared_slot: bool = False, group_top: int = 2, gate_row: bool = False, shared_slots: int = 0,
           dense: bool = True):
    """Router logits and top-k selection -> ``Routing``. Decode-sized steps (<= 64 tokens, <= 1024 pairs) run as
    ONE launch that also builds the dense routing tables; with ``norm=(weight, eps, w_offset)`` that launch first
    applies the RMSNorm to ``x`` (the raw residual stream) and ``Routing.x_normed`` is the normalised input.
    ``shared_slot``: the shared expert is stacked behind the local routed experts and gets a slot of its own that
    every token uses (weight sigmoid(x . sh_gate) when ``sh_gate`` [1, H] is given, else 1); its output rows are
    the pairs T * k .. T * k + T - 1. Larger steps use the GEMM and the selection kernel. ``gate_row`` /
    ``shared_slots``: the last row of ``w_router`` gates a shared expert stored as that many experts behind the routed ones;
    decode-sized steps give each a slot whose output rows follow the token's own pairs, larger ones return the gate.
    ``dense`` False: no dense tables (experts that do not run on the grouped GEMM)."""
    T, E = x.shape[0], w_router.shape[0] - int(gate_row)
    small = dense and T <= 64 and T * k <= 1024 and TUNE["fused_router"] and tma_ok(x, w_router)
    if not small:
        xn = None
        if norm is not None:
            xn, _ = rmsnorm(x, norm[0], norm[1], norm[2])
        logits = linear(x if xn is None else xn, w_router, out_dtype=torch.float32)
        gate = torch.empty(T, dtype=torch.float32, device=x.device) if gate_row else None
        ids, wts = router_topk(logits, k, mode, renorm, route_scale, bias, n_group, topk_group, group_top=group_top, gate=gate)
        r = Routing(ids, wts, None, xn)
        r.gate = gate
        return r
    if gate_row:
        w_router, sh_gate = w_router[:E], w_router[E]
    C = ext()
    ws = Workspace.get(x.device)
    logits = ws.buf("router_logits", (4 * 64 * 512,), torch.float32)    # one plane per column split
    ctr = ws._cache.get("router_ctr")
    if ctr is None:
        ctr = torch.zeros(4, dtype=torch.int32, device=x.device)
        ws._cache["router_ctr"] = ctr
    bn = 32 if T <= 32 else 64
    stride = slot_stride or bn
    nl = E if n_local is None else n_local
    n_slots = nl + (shared_slots or (1 if shared_slot else 0))
    dr = ws._cache.get(("dense_route", n_slots, bn, stride))
    if dr is None:
        dr = DenseRoute(n_slots, bn, x.device, stride)
        ws._cache[("dense_route", n_slots, bn, stride)] = dr
    ids = torch.empty(T, k, dtype=torch.int32, device=x.device)
    wts = torch.empty(T, k, dtype=torch.float32, device=x.device)
    xn = torch.empty_like(x) if norm is not None else None
    C.moe_route_small(x, norm[0] if norm else None, norm[1] if norm else 0.0, norm[2] if norm else 0.0, xn, w_router,
                      bias, k, ROUTER_MODES[mode], RENORM[renorm], route_scale, n_group, topk_group, logits, ids, wts,
                      stride, dr.tile_group, dr.slot_base, dr.tile_ntok, dr.meta, dr.out_rows, dr.tok_scale, ctr,
                      e_lo, nl, sh_gate.reshape(-1) if sh_gate is not None else None,
                      dr.sh_logit if sh_gate is not None else None, bool(shared_slot), ws.status, dr.active, group_top,
                      shared_slots)
    r = Routing(ids, wts, dr, xn, e_lo, nl)
    r.shared_slot, r.shared_rows = bool(shared_slot), shared_slots
    return r


class MoePlan:
    """Device buffers of one routing plan (sized for the largest step; reused every step)."""

    def __init__(self, max_tokens: int, k: int, n_local: int, bn: int, device):
        P = max_tokens * k
        i32 = dict(dtype=torch.int32, device=device)
        self.max_tokens, self.k, self.n_local, self.bn = max_tokens, k, n_local, bn
        self.max_tiles = (P + bn - 1) // bn + n_local
        self.counts = torch.zeros(n_local, **i32)
        self.offsets = torch.zeros(n_local + 1, **i32)
        self.sorted_token = torch.zeros(P, **i32)
        self.sorted_pair = torch.zeros(P, **i32)
        self.sorted_w = torch.zeros(P, dtype=torch.float32, device=device)
        self.tile_group = torch.zeros(self.max_tiles, **i32)
        self.tile_tok0 = torch.zeros(self.max_tiles, **i32)
        self.tile_ntok = torch.zeros(self.max_tiles, **i32)
        self.meta = torch.zeros(2, **i32)  # {n_tiles, n_rows}
        self.x_sorted = None
        self.h_sorted = None
        self.y_pairs = None


def _dense_ok(routing, n_groups: int, e_lo: int, ids) -> bool:
    return (routing is not None and routing.dense is not None and routing.e_lo == e_lo and routing.ids is ids
            and routing.n_local + (routing.shared_rows or int(routing.shared_slot)) == n_groups
            and (routing.shared_rows > 0 or bool(TUNE["dense_route"])))


def _dense_pairs(dr: DenseRoute, P: int, T: int, k: int, H: int, device):
    """Output rows of the down projection: one per (token, expert) pair, then one per token for the shared slot."""
    if dr.y_pairs is None or dr.y_pairs.shape[0] < P + T or dr.y_pairs.shape[1] != H:
        dr.y_pairs = torch.zeros(max(P, 64 * k) + 64, H, dtype=torch.bfloat16, device=device)
    return dr.y_pairs


class PendingCombine:
    """The weighted pair rows of a decode-sized MoE layer whose per-token sum has not run yet: the rank-partial
    result of an expert-parallel layer, handed to the reduction that follows so that it sums them inside its own
    launch (``parallel.symm.SymmComm.all_reduce_add_norm``). ``materialize`` runs the combine kernel instead."""
    __slots__ = ("y", "ids", "e_lo", "e_hi", "shared", "T", "H", "rows")

    def __init__(self, y, ids, e_lo, e_hi, shared, T, H, rows=None):
        self.y, self.ids, self.e_lo, self.e_hi, self.shared, self.T, self.H = y, ids, e_lo, e_hi, shared, T, H
        self.rows = rows or ids.shape[1]             # consecutive rows of ``y`` that make up a token

    def materialize(self, out=None):
        if out is None:
            out = torch.empty(self.T, self.H, dtype=torch.bfloat16, device=self.y.device)
        ext().moe_combine(self.y, self.ids, self.e_lo, self.e_hi, self.shared, None, None, out, None, 0.0, 0.0, None)
        return out


def _dense_combine(dr: DenseRoute, routing, ids, e_lo, T, k, H, shared, shared_gate, residual, out, norm, device,
                   defer: bool = False):
    C = ext()
    P = T * k
    y = dr.y_pairs[:P]
    if routing.shared_slot:
        # the shared expert ran as a slot of the grouped GEMMs; its gate is already applied
        shared, shared_gate = dr.y_pairs[P:P + T], None
    if defer and shared_gate is None and residual is None and norm is None:
        return PendingCombine(y, ids, e_lo, e_lo + routing.n_local, shared, T, H)
    if out is None:
        out = torch.empty(T, H, dtype=torch.bfloat16, device=device)
    if norm is None:
        C.moe_combine(y, ids, e_lo, e_lo + routing.n_local, shared, shared_gate, residual, out, None, 0.0, 0.0, None)
        return out
    normed = torch.empty(T, H, dtype=torch.bfloat16, device=device)
    C.moe_combine(y, ids, e_lo, e_lo + routing.n_local, shared, shared_gate, residual, out, norm[0], norm[1], norm[2],
                  normed)
    return out, normed


def _moe_experts_nv4(x, ids, wts, w_gate_up: "Nv4Weight", w_down: "Nv4Weight", n_ff, e_lo, shared, shared_gate,
                     residual, out, norm, routing, xq: Optional["Nv4Act"] = None, h_scale=None, defer: bool = False):
    """Routed experts on the native NVFP4 path (decode-sized steps over the dense routing): the layer input is
    quantised once (or arrives quantised as ``xq``), the gate/up GEMM re-encodes its SwiGLU output to NVFP4 in its
    epilogue (static tensor scale ``h_scale``), and the down GEMM reads that. Three launches + the combine."""
    C = ext()
    T, H = x.shape
    k = ids.shape[1]
    n_groups = w_gate_up.shape[0]
    ws = Workspace.get(x.device)
    dr = routing.dense
    P = T * k
    if xq is None:
        xq = nv4_quant_act(x, key="moe_x")
    if h_scale is None:
        h_scale = _nv4_h_scale(ws, x.device)
    rows = dr.n_slots * dr.stride
    if dr.hq is None or dr.hq[0].shape[1] * 2 != n_ff:
        dr.hq = (torch.zeros(rows, n_ff // 2, dtype=torch.uint8, device=x.device),
                 torch.zeros(C.nv4_sf_bytes(rows, n_ff), dtype=torch.uint8, device=x.device))
    hq_codes, hq_sf = dr.hq
    y_pairs = _dense_pairs(dr, P, T, k, H, x.device)
    C.wgemm_nv4(w_gate_up.view2d(), w_gate_up.sf, w_gate_up.gscale, xq.codes, xq.sf, xq.gscale, xq.stride, None, None,
                None, None, n_ff, True, n_ff, 0, dr.bn, ws.status, dr.tile_group, dr.zeros, dr.tile_ntok, dr.meta,
                dr.n_slots, 2 * n_ff, 0, dr.slot_base, hq_codes, hq_sf, h_scale)
    C.wgemm_nv4(w_down.view2d(), w_down.sf, w_down.gscale, hq_codes, hq_sf, h_scale, 0, y_pairs, None, dr.tok_scale,
                dr.out_rows, H, False, 0, 0, dr.bn, ws.status, dr.tile_group, dr.slot_base, dr.tile_ntok, dr.meta,
                dr.n_slots, H, 0, None, None, None, None)
    return _dense_combine(dr, routing, ids, e_lo, T, k, H, shared, shared_gate, residual, out, norm, x.device, defer)


class Nv4Plan:
    """Routing plan and expert-sorted NVFP4 buffers of a prompt-sized step on the native path: every expert's rows
    start on a token-tile boundary (``bn`` rows) so the tile's scale factors start where the tensor-core copy
    wants them."""

    def __init__(self, max_tokens: int, k: int, n_local: int, bn: int, H: int, n_ff: int, device):
        C = ext()
        P = max_tokens * k
        i32 = dict(dtype=torch.int32, device=device)
        u8 = dict(dtype=torch.uint8, device=device)
        self.bn = bn
        self.rows = (P + n_local * bn + 127) // 128 * 128
        self.max_tiles = (P + bn - 1) // bn + n_local
        self.counts2 = torch.zeros(2 * n_local, **i32)
        self.offsets = torch.zeros(n_local + 1, **i32)
        self.sorted_token = torch.full((self.rows,), -1, **i32)
        self.sorted_pair = torch.zeros(self.rows, **i32)
        self.sorted_w = torch.zeros(self.rows, dtype=torch.float32, device=device)
        self.tile_group = torch.zeros(self.max_tiles, **i32)
        self.tile_tok0 = torch.zeros(self.max_tiles, **i32)
        self.tile_ntok = torch.zeros(self.max_tiles, **i32)
        self.meta = torch.zeros(2, **i32)
        self.x_codes = torch.zeros(self.rows, H // 2, **u8)
        self.x_sf = torch.zeros(C.nv4_sf_bytes(self.rows, H), **u8)
        self.x_gs = torch.ones(self.rows, dtype=torch.float32, device=device)
        self.h_codes = torch.zeros(self.rows, n_ff // 2, **u8)
        self.h_sf = torch.zeros(C.nv4_sf_bytes(self.rows, n_ff), **u8)
        self.y_pairs = torch.zeros(P, H, dtype=torch.bfloat16, device=device)


def _nv4_h_scale(ws, device):
    h_scale = ws._cache.get("nv4_h_scale")
    if h_scale is None:
        h_scale = torch.tensor([NV4_H_AMAX / (6.0 * 448.0)], dtype=torch.float32, device=device)
        ws._cache["nv4_h_scale"] = h_scale
    return h_scale


def _moe_experts_nv4_sorted(x, ids, wts, w_gate_up: "Nv4Weight", w_down: "Nv4Weight", n_ff, e_lo, shared, shared_gate,
                            residual, out, norm, xq: Optional["Nv4Act"] = None):
    """Routed experts of a prompt-sized step on the native NVFP4 path: the tokens are encoded once, their codes and
    scale bytes are gathered into expert order (aligned segments), the gate/up GEMM re-encodes its SwiGLU output
    and the down GEMM scatters weighted rows to their pairs. Nothing is expanded to bf16 on the way."""
    C = ext()
    T, H = x.shape
    k = ids.shape[1]
    E_local = w_gate_up.shape[0]
    ws = Workspace.get(x.device)
    bn = TUNE["nv4_sorted_bn"]
    cap = 1024
    while cap < T:
        cap *= 2
    key = ("nv4_plan", cap, k, E_local, bn, H, n_ff)
    plan = ws._cache.get(key)
    if plan is None:
        plan = Nv4Plan(cap, k, E_local, bn, H, n_ff, x.device)
        ws._cache[key] = plan
    C.moe_plan_aligned(ids, wts, e_lo, E_local, bn, bn, plan.counts2, plan.offsets, plan.sorted_token,
                       plan.sorted_pair, plan.sorted_w, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta)
    if xq is None:
        xq = nv4_quant_act(x, key="moe_x_big")
    C.nv4_gather_rows(xq.codes, xq.sf, xq.gscale if xq.stride else None, plan.sorted_token, plan.meta[1:2],
                      plan.x_codes, plan.x_sf, plan.x_gs if xq.stride else None)
    h_scale = _nv4_h_scale(ws, x.device)
    C.wgemm_nv4(w_gate_up.view2d(), w_gate_up.sf, w_gate_up.gscale, plan.x_codes, plan.x_sf,
                plan.x_gs if xq.stride else xq.gscale, 1 if xq.stride else 0, None, None, None, None, n_ff, True, n_ff,
                0, bn, ws.status, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, 2 * n_ff,
                0, None, plan.h_codes, plan.h_sf, h_scale)
    C.wgemm_nv4(w_down.view2d(), w_down.sf, w_down.gscale, plan.h_codes, plan.h_sf, h_scale, 0, plan.y_pairs, None,
                plan.sorted_w, plan.sorted_pair, H, False, 0, 0, bn, ws.status, plan.tile_group, plan.tile_tok0,
                plan.tile_ntok, plan.meta, plan.max_tiles, H, 0, None, None, None, None)
    if out is None:
        out = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    if norm is None:
        C.moe_combine(plan.y_pairs, ids, e_lo, e_lo + E_local, shared, shared_gate, residual, out, None, 0.0, 0.0, None)
        return out
    normed = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    C.moe_combine(plan.y_pairs, ids, e_lo, e_lo + E_local, shared, shared_gate, residual, out, norm[0], norm[1],
                  norm[2], normed)
    return out, normed


# largest |SwiGLU output| the static scale of the re-encoded intermediate is laid out for (checkpoints bring their
# own calibrated input scale; this is the default for weights quantised here)
NV4_H_AMAX = 32.0


def moe_experts(x, ids, wts, w_gate_up, w_down, n_ff, e_lo=0, plan: Optional[MoePlan] = None, shared=None,
                shared_gate=None, residual=None, out=None, norm=None, routing: Optional[Routing] = None,
                defer_combine: bool = False, act: str = "silu"):
    """Routed experts over the device routing plan: plan -> gather -> grouped gate/up (+SwiGLU) ->
    grouped down (x routing weight) -> combine (+ shared expert, + residual).

    w_gate_up: [E_local, 2*n_ff, H] (``act`` "relu2": un-gated, [E_local, n_ff, H]); w_down: [E_local, H, n_ff]; ids/wts:
    [T, k]. Returns bf16 [T, H]; with ``norm=(weight, eps, w_offset)`` the combine also applies that RMSNorm and (out, normed) is returned."""
    C = ext()
    T, H = x.shape
    k = ids.shape[1]
    E_local = w_gate_up.shape[0]
    ws = Workspace.get(x.device)
    if isinstance(w_gate_up, Fp8Weight):
        return _moe_experts_fp8(x, ids, wts, w_gate_up, w_down, n_ff, e_lo, shared, shared_gate, residual, out, norm,
                                routing, defer=defer_combine)
    if isinstance(w_gate_up, Nv4Weight):
        if _dense_ok(routing, E_local, e_lo, ids):
            return _moe_experts_nv4(x, ids, wts, w_gate_up, w_down, n_ff, e_lo, shared, shared_gate, residual, out,
                                    norm, routing, xq=routing.xq, defer=defer_combine)
        wfp4_ok = H % 256 == 0 and n_ff % 256 == 0       # what the de-quantising GEMM needs of K
        if (TUNE["nv4_sorted"] and (T * k >= 64 * E_local or not wfp4_ok)
                and not (routing is not None and routing.shared_slot)):
            return _moe_experts_nv4_sorted(x, ids, wts, w_gate_up, w_down, n_ff, e_lo, shared, shared_gate, residual,
                                           out, norm, xq=routing.xq if routing is not None else None)
        # steps in between: the de-quantising grouped GEMM over the routing plan (same codes, linear scale order)
        w_gate_up, w_down = w_gate_up.as_qweight(), w_down.as_qweight()
    if routing is not None and routing.shared_slot and not _dense_ok(routing, E_local, e_lo, ids):
        raise ValueError("the routing carries a shared-expert slot that these expert weights do not have")
    gated = act != "relu2"
    n_gu = (2 if gated else 1) * n_ff                # rows of an expert in w_gate_up
    if routing is not None and routing.shared_rows and not _dense_ok(routing, E_local, e_lo, ids):
        raise ValueError("the routing carries shared experts that these expert weights do not have")
    if routing is None or not routing.shared_slot:
        n_routed = E_local
    else:
        n_routed = E_local - 1
    # expert weights as 2-D operands (+ NVFP4 block scales / tensor scales when kept in 4 bits)
    if isinstance(w_gate_up, QWeight):
        (gu2, gu_sc), gu_gs = w_gate_up.view2d(), w_gate_up.gscale
    else:
        gu2, gu_sc, gu_gs = w_gate_up.view(E_local * n_gu, H), None, None
    if isinstance(w_down, QWeight):
        (dn2, dn_sc), dn_gs = w_down.view2d(), w_down.gscale
    else:
        dn2, dn_sc, dn_gs = w_down.view(E_local * H, n_ff), None, None
    if _dense_ok(routing, E_local, e_lo, ids):
        # decode-sized step: every active expert runs over all T tokens in place (no plan, no gather)
        dr = routing.dense
        P = T * k
        if dr.h_all is None or dr.h_all.shape[1] != n_ff:
            dr.h_all = torch.zeros(dr.n_slots * dr.stride, n_ff, dtype=torch.bfloat16, device=x.device)
        kp = k + routing.shared_rows
        y_pairs = _dense_pairs(dr, T * kp, T, kp, H, x.device)
        C.wgemm(gu2, x, dr.h_all, None, None, None, n_ff, gated, n_ff if gated else 0, dr.bn, 1,
                None, None, ws.status, dr.tile_group, dr.zeros, dr.tile_ntok, dr.meta, dr.n_slots, n_gu, 0, [],
                dr.slot_base, gu_sc, gu_gs, relu2=not gated)
        C.wgemm(dn2, dr.h_all, y_pairs, None, dr.tok_scale, dr.out_rows, H, False, 0,
                dr.bn, 1, None, None, ws.status, dr.tile_group, dr.slot_base, dr.tile_ntok, dr.meta, dr.n_slots, H, 0, [],
                None, dn_sc, dn_gs)
        if routing.shared_rows:
            if not defer_combine or shared is not None or residual is not None or norm is not None:
                raise NotImplementedError("shared experts among a token's pairs are summed by the step that follows")
            return PendingCombine(y_pairs[:T * kp], ids, e_lo, e_lo + routing.n_local, None, T, H, kp)
        return _dense_combine(dr, routing, ids, e_lo, T, k, H, shared, shared_gate, residual, out, norm, x.device,
                              defer_combine)
    E_local = n_routed
    if plan is None:
        bn = 32 if T * k <= 32 * E_local else (64 if T * k <= 64 * E_local else 128)
        key = ("moe_plan", T, k, E_local, bn, H, n_ff)
        plan = ws._cache.get(key)
        if plan is None:
            plan = MoePlan(T, k, E_local, bn, x.device)
            ws._cache[key] = plan
    P = T * k
    bn = plan.bn
    if (plan.x_sorted is None or plan.x_sorted.shape[0] < P + bn or plan.x_sorted.shape[1] != H
            or plan.h_sorted.shape[1] != n_ff):
        # padded by one tile so a tile that starts near the end stays inside the tensor map's rows
        plan.x_sorted = torch.zeros(P + bn, H, dtype=torch.bfloat16, device=x.device)
        plan.h_sorted = torch.zeros(P + bn, n_ff, dtype=torch.bfloat16, device=x.device)
        plan.y_pairs = torch.zeros(P, H, dtype=torch.bfloat16, device=x.device)
    if P <= 1024 and E_local <= 512 and TUNE["fused_plan"]:
        # decode-sized step: plan and gather in one launch
        C.moe_plan_gather(ids, wts, e_lo, E_local, bn, plan.counts, plan.offsets, plan.sorted_token,
                          plan.sorted_pair, plan.sorted_w, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta,
                          x, plan.x_sorted)
    else:
        C.moe_plan(ids, wts, e_lo, E_local, bn, plan.counts, plan.offsets, plan.sorted_token, plan.sorted_pair,
                   plan.sorted_w, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta)
        C.gather_rows(x, plan.sorted_token, plan.meta[1:2], plan.x_sorted[:P])
    C.wgemm(gu2, plan.x_sorted, plan.h_sorted, None, None, None, n_ff, gated, n_ff if gated else 0, bn, 1, None, None, ws.status,
            plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, n_gu, 0, [], None,
            gu_sc, gu_gs, relu2=not gated)
    C.wgemm(dn2, plan.h_sorted, plan.y_pairs, None, plan.sorted_w, plan.sorted_pair, H, False, 0, bn, 1, None, None,
            ws.status, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, H, 0, [], None,
            dn_sc, dn_gs)
    if defer_combine == "pairs":
        return PendingCombine(plan.y_pairs, ids, e_lo, e_lo + E_local, None, T, H)
    if out is None:
        out = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    if norm is None:
        C.moe_combine(plan.y_pairs, ids, e_lo, e_lo + E_local, shared, shared_gate, residual, out, None, 0.0, 0.0, None)
        return out
    normed = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    C.moe_combine(plan.y_pairs, ids, e_lo, e_lo + E_local, shared, shared_gate, residual, out, norm[0], norm[1],
                  norm[2], normed)
    return out, normed


def moe_experts_plain(x, ids, wts, w_gate_up, w_down, n_ff, act="silu", e_lo=0, shared=None, shared_gate=None,
                      residual=None, norm=None, defer_combine=False):
    """Routed experts on the FMA units over the same routing plan (fp32 models, unaligned bf16 shapes; all experts
    local, without a shared one). With ``defer_combine`` the weighted pair rows are handed on."""
    gated = act != "relu2"
    n_gu = (2 if gated else 1) * n_ff
    if e_lo or shared is not None or residual is not None or norm is not None or w_gate_up.shape[1] != n_gu:
        raise NotImplementedError("plain experts: all local, no shared expert, residual or norm")
    C = ext()
    T, H = x.shape
    k, E = ids.shape[1], w_gate_up.shape[0]
    P, bn = T * k, 32
    ws = Workspace.get(x.device)
    key = ("moe_plan_plain", T, k, E)
    plan = ws._cache.get(key)
    if plan is None:
        plan = ws._cache[key] = MoePlan(T, k, E, bn, x.device)
    C.moe_plan(ids, wts, 0, E, bn, plan.counts, plan.offsets, plan.sorted_token, plan.sorted_pair, plan.sorted_w,
               plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta)
    xs = x.index_select(0, plan.sorted_token)
    h = torch.empty(P, n_ff, dtype=x.dtype, device=x.device)
    y = torch.empty(P, H, dtype=x.dtype, device=x.device)
    C.sgemm(w_gate_up.view(E * n_gu, H), xs, h, None, None, None, n_ff, gated, n_ff if gated else 0, GATE_ACTS[act],
            plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, n_gu, P, None)
    C.sgemm(w_down.view(E * H, n_ff), h, y, None, plan.sorted_w, plan.sorted_pair, H, False, 0, 0, plan.tile_group,
            plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, H, P, None)
    if defer_combine:
        return PendingCombine(y, ids, 0, E, None, T, H)
    return y.view(T, k, H).sum(1, dtype=torch.float32).to(x.dtype)


def _moe_experts_fp8(x, ids, wts, w_gate_up, w_down, n_ff, e_lo, shared, shared_gate, residual, out, norm, routing,
                     defer: bool = False):
    """Routed experts with block-scaled FP8 weights: the same two grouped GEMMs in FP8 mode; activations (the
    layer input and the SwiGLU output) are quantised per row and 128 columns before each of them."""
    C = ext()
    T, H = x.shape
    k = ids.shape[1]
    E_local = w_gate_up.shape[0]
    ws = Workspace.get(x.device)
    gu2, gu_s = w_gate_up.view2d()
    dn2, dn_s = w_down.view2d()
    P = T * k
    if out is None:
        out = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    if _dense_ok(routing, E_local, e_lo, ids):
        dr = routing.dense
        if dr.h_all is None or dr.h_all.shape[1] != n_ff:
            dr.h_all = torch.zeros(dr.n_slots * dr.stride, n_ff, dtype=torch.bfloat16, device=x.device)
        y_pairs = _dense_pairs(dr, P, T, k, H, x.device)
        x8, xs = _fp8_parts(routing.xq) if isinstance(routing.xq, Fp8Act) else fp8_quant_act(x)
        if TUNE["fp8_fused_quant"] and n_ff % 128 == 0:
            # the gate/up epilogue encodes the activated rows itself (rows past a slot's tokens stay zero bytes)
            if dr.h8 is None or dr.h8.shape[1] != n_ff:
                dr.h8 = torch.zeros(dr.n_slots * dr.stride, n_ff, dtype=torch.uint8, device=x.device)
                dr.h8_scale = torch.ones(dr.n_slots * dr.stride, n_ff // 128, dtype=torch.float32, device=x.device)
            h8, hs = dr.h8, dr.h8_scale
            C.wgemm_fp8_q(gu2, gu_s, x8, xs, dr.h_all, None, None, None, n_ff, True, n_ff, dr.bn, 1, None, None,
                          ws.status, dr.tile_group, dr.zeros, dr.tile_ntok, dr.meta, dr.n_slots, 2 * n_ff, 0,
                          dr.slot_base, h8, hs)
        else:
            C.wgemm_fp8(gu2, gu_s, x8, xs, dr.h_all, None, None, None, n_ff, True, n_ff, dr.bn, 1, None, None,
                        ws.status, dr.tile_group, dr.zeros, dr.tile_ntok, dr.meta, dr.n_slots, 2 * n_ff, 0, dr.slot_base)
            h8, hs = fp8_quant_act(dr.h_all)
        C.wgemm_fp8(dn2, dn_s, h8, hs, y_pairs, None, dr.tok_scale, dr.out_rows, H, False, 0, dr.bn, 1, None, None,
                    ws.status, dr.tile_group, dr.slot_base, dr.tile_ntok, dr.meta, dr.n_slots, H, 0, None)
        return _dense_combine(dr, routing, ids, e_lo, T, k, H, shared, shared_gate, residual, out, norm, x.device,
                              defer=defer)
    if True:
        bn = 32 if P <= 32 * E_local else 64
        key = ("moe_plan", T, k, E_local, bn, H, n_ff)
        plan = ws._cache.get(key)
        if plan is None:
            plan = MoePlan(T, k, E_local, bn, x.device)
            ws._cache[key] = plan
        if (plan.x_sorted is None or plan.x_sorted.shape[0] < P + bn or plan.x_sorted.shape[1] != H
                or plan.h_sorted.shape[1] != n_ff):
            plan.x_sorted = torch.zeros(P + bn, H, dtype=torch.bfloat16, device=x.device)
            plan.h_sorted = torch.zeros(P + bn, n_ff, dtype=torch.bfloat16, device=x.device)
            plan.y_pairs = torch.zeros(P, H, dtype=torch.bfloat16, device=x.device)
        C.moe_plan(ids, wts, e_lo, E_local, bn, plan.counts, plan.offsets, plan.sorted_token, plan.sorted_pair,
                   plan.sorted_w, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta)
        C.gather_rows(x, plan.sorted_token, plan.meta[1:2], plan.x_sorted[:P])
        x8, xs = fp8_quant_act(plan.x_sorted)
        C.wgemm_fp8(gu2, gu_s, x8, xs, plan.h_sorted, None, None, None, n_ff, True, n_ff, bn, 1, None, None, ws.status,
                    plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, 2 * n_ff, 0, None)
        h8, hs = fp8_quant_act(plan.h_sorted)
        C.wgemm_fp8(dn2, dn_s, h8, hs, plan.y_pairs, None, plan.sorted_w, plan.sorted_pair, H, False, 0, bn, 1, None,
                    None, ws.status, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta, plan.max_tiles, H, 0,
                    None)
        y = plan.y_pairs
    if norm is None:
        C.moe_combine(y, ids, e_lo, e_lo + E_local, shared, shared_gate, residual, out, None, 0.0, 0.0, None)
        return out
    normed = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    C.moe_combine(y, ids, e_lo, e_lo + E_local, shared, shared_gate, residual, out, norm[0], norm[1], norm[2], normed)
    return out, normed


def token_logprobs(logits, chosen, n_top: int = 0):
    """(log-probability of chosen[r] in row r, top-n token ids [R, n], their log-probabilities [R, n])."""
    C = ext()
    R = logits.shape[0]
    lp = torch.empty(R, dtype=torch.float32, device=logits.device)
    ids = torch.empty(R, max(n_top, 1), dtype=torch.int32, device=logits.device)
    tl = torch.empty(R, max(n_top, 1), dtype=torch.float32, device=logits.device)
    C.token_logprobs(logits, chosen.int(), n_top, lp, ids, tl)
    return lp, ids[:, :n_top], tl[:, :n_top]


def spec_accept(target, cu, draft, n_draft):
    """Greedy acceptance on the device: (accepted drafts per sequence, the token after the accepted prefix,
    flag: some draft was rejected)."""
    C = ext()
    B = draft.shape[0]
    acc = torch.empty(B, dtype=torch.int32, device=target.device)
    bonus = torch.empty(B, dtype=torch.int32, device=target.device)
    rej = torch.zeros(1, dtype=torch.int32, device=target.device)
    C.spec_accept(target.int(), cu.int(), draft.int().contiguous(), n_draft.int(), acc, bonus, rej)
    return acc, bonus, rej


def argmax(logits, out=None, out_val=None):
    C = ext()
    rows, V = logits.shape
    ws = Workspace.get(logits.device)
    nblk = max(1, min(64, (V + 4095) // 4096))
    pv = ws.buf("argmax_v", (rows * nblk,), torch.float32)
    pi = ws.buf("argmax_i", (rows * nblk,), torch.int32)
    if out is None:
        out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    C.argmax(logits, pv, pi, out, out_val)
    return out


def sample(logits, temperature, top_k, top_p, min_p, seeds, steps, out=None):
    C = ext()
    rows, V = logits.shape
    ws = Workspace.get(logits.device)
    scratch = ws.buf("sample", (rows * V,), torch.float32)
    if out is None:
        out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    C.sample(logits, temperature, top_k, top_p, min_p, seeds, steps, scratch, out)
    return out


def causal_conv1d_silu(x, w, bias, conv_state, cu_seq, slots, write_state=True, out=None, max_len=None, in_bias=None,
                       silu: bool = True):
    """``max_len``: longest sequence of the step when known on the host; prompt-sized steps (>= 64 rows per
    sequence) run the token-parallel kernel."""
    C = ext()
    if out is None:
        out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    if x.dtype != torch.bfloat16 or not 2 <= w.shape[1] <= 8:
        C.conv_silu_any(x, w, bias, conv_state, cu_seq, slots, out, bool(write_state), in_bias, bool(silu))
        return out
    T, n = x.shape[0], max(1, slots.numel())
    if max_len is None:
        max_len = T if T >= 64 * n else 0          # without the host figure: only clearly prompt-sized steps
    C.conv1d_silu(x, w, bias, conv_state, cu_seq, slots, out, write_state, int(max_len) if max_len >= 64 else 0, in_bias,
                  bool(silu))
    return out


def gdn_gates(a, b, A, dt_bias):
    C = ext()
    g = torch.empty(a.shape, dtype=torch.float32, device=a.device)
    beta = torch.empty_like(g)
    C.gdn_gates(a, b, A, dt_bias, g, beta)
    return g, beta


def gdn_chunk_plan(cu_host, device):
    """Host-side tables of the chunked scan for one step: 128-token blocks and per-sequence chunk ranges."""
    blk_t0, blk_n, seq_blk0, seq_nchunk, seq_t0, seq_len = [], [], [], [], [], []
    for i in range(len(cu_host) - 1):
        t0, n = cu_host[i], cu_host[i + 1] - cu_host[i]
        seq_blk0.append(len(blk_t0))
        seq_nchunk.append((n + 63) // 64)
        seq_t0.append(t0)
        seq_len.append(n)
        for b in range(0, n, 128):
            blk_t0.append(t0 + b)
            blk_n.append(min(128, n - b))
    i32 = dict(dtype=torch.int32, device=device)
    return tuple(torch.tensor(v, **i32) for v in (blk_t0, blk_n, seq_blk0, seq_nchunk, seq_t0, seq_len))


def gdn_chunked(qkv, g, beta, state, cu_host, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps=1e-6,
                write_state=True, out=None):
    """Gated delta rule over prompt-sized rows on the tensor cores (64-token chunks, ``csrc/gdn_chunk_sm100.cu``).
    ``cu_host``: the sequence boundaries as a Python list. Heads of 128 x 128 only."""
    C = ext()
    T = qkv.shape[0]
    ws = Workspace.get(qkv.device)
    blk_t0, blk_n, seq_blk0, seq_nchunk, seq_t0, seq_len = gdn_chunk_plan(cu_host, qkv.device)
    nb = int(blk_t0.numel())
    need = C.gdn_chunk_scratch_bytes(nb, n_v)
    scratch = ws._cache.get("gdn_chunk_scratch")
    if scratch is None or scratch.numel() < need:
        scratch = torch.empty(need, dtype=torch.uint8, device=qkv.device)
        ws._cache["gdn_chunk_scratch"] = scratch
    if out is None:
        out = torch.empty(T, n_v, dv, dtype=torch.bfloat16, device=qkv.device)
    C.gdn_chunk(qkv, g.contiguous(), beta.contiguous(), state, blk_t0, blk_n, seq_blk0, seq_nchunk, seq_t0, seq_len,
                slots, n_k, n_v, dk, dv, bool(tiled_heads), scale, l2_eps, out, bool(write_state), scratch, ws.status)
    return out


def gdn_recurrent(qkv, g, beta, state, cu_seq, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps=1e-6,
                  write_state=True, out=None, cu_host=None):
    C = ext()
    T = qkv.shape[0]
    # prompt chunks (many rows per sequence): the chunked tensor-core scan when the heads are 128 x 128, else the
    # column-per-thread kernel; decode rows run the state-streaming one
    prompt_rows = T >= 16 * max(1, slots.numel())
    if prompt_rows and dk == 128 and dv == 128 and T >= 64 and TUNE["gdn_chunk"] and qkv.stride(0) % 8 == 0:
        if cu_host is None:
            cu_host = cu_seq.tolist()
        return gdn_chunked(qkv, g, beta, state, cu_host, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps,
                           write_state, out)
    if out is None:
        out = torch.empty(T, n_v, dv, dtype=torch.bfloat16, device=qkv.device)
    C.gdn_recurrent(qkv, g, beta, state, cu_seq, slots, n_k, n_v, dk, dv, tiled_heads, scale, l2_eps, out,
                    write_state, True, prompt_rows)
    return out


def gdn_decode_fused_ok(n_k, n_v, dk, dv, conv_k) -> bool:
    return dk == dv and dk in (64, 128) and conv_k == 4 and n_k > 0 and n_v % n_k == 0 and n_v // n_k <= 4


def gdn_decode_fused(proj, conv_w, conv_state, A, dt_bias, norm_w, eps, act, state, slots, n_k, n_v, dk, dv,
                     tiled_heads, scale, l2_eps=1e-6, out=None):
    """One launch for the decode step of a Gated DeltaNet layer: conv + SiLU with history update, gates, delta rule
    with state update, gated RMS norm. ``proj`` [n_seqs, q|k|v|z|b|a] is the fused input projection of the step's
    tokens (one per sequence, in sequence order). Returns bf16 [n_seqs, n_v * dv]."""
    C = ext()
    n = slots.numel()
    if out is None:
        out = torch.empty(n, n_v * dv, dtype=torch.bfloat16, device=proj.device)
    C.gdn_decode_fused(proj, conv_w, conv_state, A, dt_bias, norm_w, eps, 0 if act == "silu" else 1, state, slots,
                       n_k, n_v, dk, dv, bool(tiled_heads), scale, l2_eps, out)
    return out


def mamba2_scan_ok(nh: int, hd: int, ng: int, ds: int) -> bool:
    """Head shapes the Mamba-2 kernel's thread layout covers (256 / hd threads per state row, <= 32 columns each)."""
    if hd <= 0 or hd > 256 or 256 % hd or hd & (hd - 1) or nh % max(ng, 1):
        return False
    W = 256 // hd
    return W <= 32 and ds % W == 0 and ds // W <= 32


def mamba2_scan(xbc, dt_raw, z, A, D, dt_bias, state, cu_seq, slots, nh, hd, ng, ds, write_state=True, out=None):
    """Mamba-2 recurrence over the step's tokens: xbc [T, nh*hd + 2*ng*ds] = x | B | C after the causal conv, dt_raw
    [T, nh], z [T, nh*hd] (bf16, row slices allowed), fp32 state [slots, nh, hd, ds] updated in place. Returns
    (S C + D x) * silu(z) as bf16 [T, nh*hd]."""
    C = ext()
    T = xbc.shape[0]
    if out is None:
        out = torch.empty(T, nh * hd, dtype=torch.bfloat16, device=xbc.device)
    if T == 0:
        return out
    C.mamba2_scan(xbc, dt_raw, z, A.float(), D.float(), dt_bias.float(), state, cu_seq, slots, nh, hd, ng, ds, out,
                  bool(write_state))
    return out


def hyper_start(table, ids, streams: int, in_w, norm_w, eps, w_offset=0.0):
    """Streams [T, S, H] fp32 from the embedding and the normed input of the first sublayer, in one launch."""
    T = table.shape[0] if ids is None else ids.numel()
    X = torch.empty(T, streams, table.shape[1], dtype=torch.float32, device=table.device)
    h = torch.empty(T, table.shape[1], dtype=table.dtype, device=table.device)
    ext().hyper_step(None, X, table, ids, None, 0.0, 1, None, 0.0, None, None, in_w, norm_w, eps, w_offset, h)
    return X, h


def hyper_step(X, terms, mix, out_w, in_w, norm_w, eps, w_offset=0.0):
    """X (fp32 streams) updated in place behind a sublayer, and the normed input of the next one. A ``PendingCombine``
    term is summed over its weighted expert rows inside the launch."""
    (y0, c0), (y1, c1) = (list(terms) + [(None, 0.0)])[:2]
    rows = 1
    if isinstance(y0, PendingCombine):
        rows, y0 = y0.rows, y0.y
    h = torch.empty(X.shape[0], X.shape[2], dtype=y0.dtype, device=X.device)
    ext().hyper_step(X, X, None, None, y0, c0, rows, y1, c1, mix, out_w, in_w, norm_w, eps, w_offset, h)
    return X, h


def prenorm_step(x, terms, mult, norm_w, eps, w_offset=0.0, raw=None, start=None, dtype=None, x_out=None):
    """x (fp32 [T, H]) updated in place by mult * (sum of scale * tensor over ``terms``), and its norm in the activation type
    (``norm_w`` None: none); ``raw`` takes x itself in the activation type. ``start`` = (embedding table, ids or None, norm
    weight or None) begins a step. Returns (x, norm)."""
    table = ids = pre_w = None
    x_in = x
    if start is not None:
        table, ids, pre_w = start
        T = table.shape[0] if ids is None else ids.numel()
        x, dtype = torch.empty(T, table.shape[1], dtype=torch.float32, device=table.device) if x_out is None else x_out, table.dtype
    (y0, c0), (y1, c1) = (list(terms) + [(None, 0.0), (None, 0.0)])[:2]
    rows = 1
    if isinstance(y0, PendingCombine):
        rows, y0 = y0.rows, y0.y
    h = torch.empty(x.shape, dtype=dtype, device=x.device) if norm_w is not None else None
    if x.shape[0]:
        ext().prenorm_step(x_in, x, table, ids, pre_w, y0, c0 * mult, rows, y1, c1 * mult, norm_w, eps, w_offset, h, raw)
    return x, h


DEPTH_AHEAD = 3              # layers for which a pass over all earlier results sums up ahead (csrc/layers.h)


class DepthHistory:
    """The embedding output and the results of the layers, [layers + 1, T, H] float32, and the sums over them that a pass of
    ``depth_step`` left for the layers behind it."""
    __slots__ = ("X", "ahead")

    def __init__(self, X):
        self.X, self.ahead = X, None


def depth_step(x, hist, i: int, y1, g1, b1, y2, g2, b2, y2_b, coefs, norm_w, eps, w_offset=0.0, rows=None):
    """``reference.depth_step`` in one launch (``csrc/depth_step.cu``). ``x`` is updated in place unless it is an entry of
    ``hist`` or only ``rows`` are wanted; the last layer's result is not kept. One layer in ``DEPTH_AHEAD`` + 1 reads all
    earlier results, and sums them up for the layers behind it too."""
    y2_rows = 1
    if isinstance(y2, PendingCombine):
        y2_rows, y2 = y2.rows, y2.y
    n = x.shape[0] if rows is None else rows.numel()
    own = rows is not None or (hist is not None and x.data_ptr() == hist.X.data_ptr())
    x_out = torch.empty(n, x.shape[1], dtype=torch.float32, device=x.device) if own else x
    h = torch.empty(n, x.shape[1], dtype=y1.dtype, device=x.device)
    if n == 0:
        return x_out, h
    X = part = ahead = None
    first, keep, r = 0, False, i % (DEPTH_AHEAD + 1)
    if hist is not None:
        X = hist.X
        keep = i + 2 < X.shape[0]
        if r:
            part, first, coefs = hist.ahead[r - 1], i - r + 2, coefs[:1]
        elif len(coefs) > 1:
            ahead = hist.ahead = torch.empty(len(coefs) - 1, *x.shape, dtype=torch.float32, device=x.device)
    ext().depth_step(x, x_out, X, i, first, part, keep, y1, g1, b1, y2, y2_rows, g2, b2, y2_b, coefs or [], ahead, norm_w, eps,
                     w_offset, h, rows)
    return x_out, h


def qkv_conv_append(proj, in_b, conv_w, conv_state, cu_seq, state_slots, q_norm, k_norm, norm_over, eps, rot, layout, positions,
                    slots, k_cache, v_cache, heads: int, write_state=True, max_len=None):
    """Bias, short convolution, norms, rotation of a q | k | v projection and the append to the cache (``csrc/qkv_conv.cu``);
    returns the queries [T, heads, dk]."""
    T = proj.shape[0]
    q = torch.empty(T, heads, k_cache.shape[3], dtype=proj.dtype, device=proj.device)
    ext().qkv_conv_append(proj, in_b, conv_w, conv_state, cu_seq, state_slots, q_norm, k_norm, norm_over == "all", eps, rot,
                          layout == "half", positions, slots, q, k_cache, v_cache, T if max_len is None else int(max_len),
                          bool(write_state))
    return q


DELTA_SCRATCH = 256 << 20    # bytes of block records a slice of a long step may take


def channel_delta(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H, G, dk, dv, write_state=True,
                  max_len=None, cu_host=None, out=None):
    """Gated delta rule with a decay per key channel over the step's tokens, convolution included
    (``csrc/channel_delta.cu``); state [slots, H, dv, dk] fp32 updated in place. Returns [T, H * dv]."""
    C = ext()
    T, n = qkv.shape[0], slots.numel()
    if out is None:
        out = torch.empty(T, H * dv, dtype=qkv.dtype, device=qkv.device)
    if T == 0:
        return out
    ws = Workspace.get(qkv.device)
    per = C.channel_delta_record_floats(H, dk, dv, qkv.dtype == torch.float32)
    need = (T + 3) // 4 + 2 * n + 2                # records of the whole step
    if write_state:                                # a long step may run in slices of at least 64 tokens
        need = min(need, max(DELTA_SCRATCH // (4 * per), 2 * n + 18))
    rec = ws._cache.get("channel_delta_rec")
    if rec is None or rec.numel() < need * per:
        rec = ws._cache["channel_delta_rec"] = torch.empty(need * per, dtype=torch.float32, device=qkv.device)
    C.channel_delta(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H, G, dk, dv, out, bool(write_state),
                    rec, ws.status)
    return out


def channel_delta_decode(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H, G, dk, dv, gate, norm_w, eps,
                         out=None):
    """Decode step of ``channel_delta`` (one token per sequence) with the norm per head and sigmoid(gate) behind it, in one
    launch."""
    n = slots.numel()
    ws = Workspace.get(qkv.device)
    ctr = ws._cache.get("delta_ctr")
    if ctr is None or ctr.numel() < n * G:
        ctr = ws._cache["delta_ctr"] = torch.zeros(max(n * G, 16384), dtype=torch.int32, device=qkv.device)
    if out is None:
        out = torch.empty(n, H * dv, dtype=qkv.dtype, device=qkv.device)
    ext().channel_delta_decode(qkv, conv_w, conv_state, a_raw, A, dt_bias, b_raw, state, cu_seq, slots, H, G, dk, dv, gate, norm_w,
                               eps, ctr, out)
    return out


def head_norm_gate(o, gate, w, eps, heads: int, out=None):
    """RMS norm of each head of o [T, heads * d], times w [d], times sigmoid(gate)."""
    if out is None:
        out = torch.empty(o.shape, dtype=o.dtype, device=o.device)
    ext().head_norm_gate(o, gate, w, eps, heads, out)
    return out


LINEAR_CHUNK_MIN = 48        # longest portion of a step from which the chunked scan runs
LINEAR_CHUNK_SHORT = 8       # ... and up to which its shorter portions stay on the streaming kernel


def _linear_chunk_tables(ws, cu_host, device, size: int = 128):
    """chunk_t0 | chunk_n | chunk_seq | seq_chunk0 | seq_nchunk of a step (chunks of ``size`` tokens; short portions have
    none); kept for the step's other layers. Returns (tables, chunks, whether there are short portions)."""
    key = tuple(cu_host)
    name = ("linear_chunk_tables", size)
    last = ws._cache.get(name)
    if last is not None and last[0] == key:
        return last[1:]
    t0, n, sq, first, cnt = [], [], [], [], []
    for i in range(len(cu_host) - 1):
        first.append(len(t0))
        if cu_host[i + 1] - cu_host[i] <= LINEAR_CHUNK_SHORT:
            cnt.append(0)
            continue
        for b in range(cu_host[i], cu_host[i + 1], size):
            t0.append(b)
            n.append(min(size, cu_host[i + 1] - b))
            sq.append(i)
        cnt.append(len(t0) - first[-1])
    tab = torch.tensor(t0 + n + sq + first + cnt, dtype=torch.int32, device=device)
    short = any(c == 0 for c in cnt)
    ws._cache[name] = (key, tab, len(t0), short)
    return tab, len(t0), short


def linear_scan(q, k, v, state, cu_seq, slots, H, G, N, P, decay=None, silu_in=False, dt=None, dt_bias=None, A=None,
                D=None, z=None, write_state=True, max_len=None, cu_host=None, out=None, chunked=None):
    """Decayed linear-attention state over the step's tokens (constant or selective decay), state [slots, H, P, N] fp32
    updated in place. bf16 prompts run in 128-token chunks on the tensor cores (``csrc/linear_scan_sm100.cu``), decode
    rows, short portions and fp32 on the streaming kernel (``csrc/linear_scan.cu``). ``chunked`` forces the choice."""
    C = ext()
    if out is None:
        out = torch.empty(q.shape[0], H * P, dtype=q.dtype, device=q.device)
    args = (q, k, v, bool(silu_in), decay, dt, dt_bias, A, D, z, state, cu_seq, slots, H, G, N, P, out, bool(write_state))
    if chunked is None:
        chunked = (q.dtype == torch.bfloat16 and cu_host is not None and (max_len or 0) >= LINEAR_CHUNK_MIN
                   and C.linear_chunk_ok(N, P))
    if not chunked:
        C.linear_scan(*args, 0)
        return out
    ws = Workspace.get(q.device)
    tab, n_chunks, short = _linear_chunk_tables(ws, cu_host if cu_host is not None else cu_seq.tolist(), q.device)
    if short or n_chunks == 0:           # single tokens and the like beside prompts
        C.linear_scan(*args, LINEAR_CHUNK_SHORT)
    if n_chunks == 0:
        return out
    need = C.linear_chunk_scratch_bytes(n_chunks, H, N, P)
    scratch = ws._cache.get("linear_chunk_scratch")
    if scratch is None or scratch.numel() < need:
        scratch = ws._cache["linear_chunk_scratch"] = torch.empty(need, dtype=torch.uint8, device=q.device)
    C.linear_chunk(*args, tab, n_chunks, scratch, ws.status)
    return out


def forget_scan(q, f, v, f_b, lower, state, cu_seq, slots, H, N, P, norm_w, eps, scale=1.0, write_state=True, max_len=None,
                cu_host=None, out=None, chunked=None):
    """HGRN2 state over the step's tokens with the norm per head behind it, state [slots, H, P, N] fp32 updated in place. bf16
    prompts run in 128-token chunks on the tensor cores (``csrc/forget_scan_sm100.cu``), decode rows, short portions and fp32
    on the streaming kernel (``csrc/forget_scan.cu``). ``chunked`` forces the choice."""
    C = ext()
    if out is None:
        out = torch.empty(q.shape[0], H * P, dtype=q.dtype, device=q.device)
    args = (q, f, v, f_b, lower, state, cu_seq, slots, H, N, P, norm_w, float(eps), float(scale), out, bool(write_state))
    if chunked is None:
        chunked = (q.dtype == torch.bfloat16 and cu_host is not None and (max_len or 0) >= LINEAR_CHUNK_MIN
                   and C.forget_chunk_ok(N, P))
    if not chunked:
        C.forget_scan(*args, 0)
        return out
    ws = Workspace.get(q.device)
    tab, n_chunks, short = _linear_chunk_tables(ws, cu_host if cu_host is not None else cu_seq.tolist(), q.device)
    if short or n_chunks == 0:           # single tokens and the like beside prompts
        C.forget_scan(*args, LINEAR_CHUNK_SHORT)
    if n_chunks == 0:
        return out
    need = C.forget_chunk_scratch_bytes(n_chunks, H, N, P)
    scratch = ws._cache.get("linear_chunk_scratch")
    if scratch is None or scratch.numel() < need:
        scratch = ws._cache["linear_chunk_scratch"] = torch.empty(need, dtype=torch.uint8, device=q.device)
    C.forget_chunk(*args, tab, n_chunks, scratch, ws.status)
    return out


def ssd_decode(xbc, conv_w, conv_b, conv_state, dt, dt_bias, A, D, z, state, cu_seq, slots, H, G, N, P, out=None):
    """Decode step of a Mamba-2 mixer in one launch (one token per sequence): convolution with history update, step
    size, state update, skip and silu(z) gate. ``xbc``: x | B | C columns of the input projection."""
    n = slots.numel()
    ws = Workspace.get(xbc.device)
    ctr = ws._cache.get("ssd_ctr")
    if ctr is None or ctr.numel() < n * G:
        ctr = ws._cache["ssd_ctr"] = torch.zeros(max(n * G, 4096), dtype=torch.int32, device=xbc.device)
    if out is None:
        out = torch.empty(n, H * P, dtype=xbc.dtype, device=xbc.device)
    ext().ssd_decode(xbc, conv_w, conv_b, conv_state, dt, dt_bias, A, D, z, state, cu_seq, slots, H, G, N, P, ctr, out)
    return out


def group_norm_gate(y, gate, w, eps, groups: int = 1, out=None):
    """RMS norm of each of ``groups`` equal parts of a row, times w, times sigmoid(gate) when a gate is given."""
    if out is None:
        out = torch.empty(y.shape, dtype=y.dtype, device=y.device)
    ext().group_norm_gate(y, gate, w, eps, groups, out)
    return out


def softcap(logits, scale: float, cap: float):
    """cap * tanh(logits * scale / cap) in place, float32."""
    ext().softcap(logits, float(scale), float(cap))
    return logits


def resid_tokens(rows: int, max_len: int, width: int, groups: int) -> int:
    """Tokens per CTA of ``resid_step``: as few as give one wave of CTAs (about 12 warps per SM, a warp per 512 columns of
    a group), so that the rows recomputed in front of a tile cost little in long runs and short ones still fill the SMs."""
    if max_len <= 1:
        return 1
    warps = groups * -(-(width // groups) // 512)
    return max(4, min(32, -(-rows * warps // (12 * NUM_SMS))))


def resid_step(x, y, post_w, norm_w, groups: int, eps: float, conv=None, start=None, max_len=None):
    """x + norm(y) into a new buffer, its norm and the input convolution behind it, in one launch. ``start`` = (embedding
    table, ids or None, scale) begins a step. Returns (x, input of the next sublayer)."""
    if start is None:
        table = ids = None
        scale, xo, h = 1.0, torch.empty_like(x), torch.empty(x.shape, dtype=y.dtype, device=x.device)
    else:
        table, ids, scale = start
        T = table.shape[0] if ids is None else ids.numel()
        xo = torch.empty(T, table.shape[1], dtype=torch.float32, device=table.device)
        h = torch.empty(T, table.shape[1], dtype=table.dtype, device=table.device)
    taps, hist, cu, slots, write = conv if conv is not None else (None, None, None, None, False)
    rows = xo.shape[0]
    if rows == 0:
        return xo, h
    max_len = rows if max_len is None else max_len
    tok = 1
    if taps is not None:
        tok = max(resid_tokens(rows, max_len, xo.shape[1], groups), min(taps.shape[0] - 1, max_len))
    ext().resid_step(x, xo, table, ids, float(scale), y, post_w, norm_w, groups, eps, taps, hist, cu, slots, bool(write),
                     int(max_len), tok, h)
    return xo, h


def block_gates(u, w, blocks: int):
    """Block-diagonal product of u [T, W] with w [blocks * n, W / blocks], float32 [T, blocks * n]."""
    T, d, n = u.shape[0], w.shape[1], w.shape[0] // blocks
    out = torch.empty(T * blocks, n, dtype=torch.float32, device=u.device)
    return head_linear(u, w, blocks, n, n, d, d, out).view(T, blocks * n)


DIAG_CHUNK = 64              # tokens per chunk of the diagonal recurrence


def gated_recurrence(u, gates, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks: int, write_state=True, max_len=None,
                     cu_host=None, out=None, chunked=None):
    """RG-LRU over the step's tokens (``reference.gated_recurrence``). Prompts run in chunks, short portions token by
    token; ``chunked`` forces the choice. The chunked form overwrites ``gates``."""
    C = ext()
    if out is None:
        out = torch.empty(u.shape, dtype=u.dtype, device=u.device)
    args = (u, gates, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks, out, bool(write_state))
    if chunked is None:
        chunked = cu_host is not None and (max_len or 0) >= LINEAR_CHUNK_MIN
    if not chunked:
        C.diag_scan(*args, 0, None, 0, None)
        return out
    ws = Workspace.get(u.device)
    tab, n_chunks, short = _linear_chunk_tables(ws, cu_host if cu_host is not None else cu_seq.tolist(), u.device, DIAG_CHUNK)
    if short or n_chunks == 0:
        C.diag_scan(*args, LINEAR_CHUNK_SHORT, None, 0, None)
    if n_chunks:
        need = n_chunks * 2 * u.shape[1]
        ends = ws._cache.get("diag_chunk_ends")
        if ends is None or ends.numel() < need:
            ends = ws._cache["diag_chunk_ends"] = torch.empty(need, dtype=torch.float32, device=u.device)
        C.diag_scan(*args, 0, tab, n_chunks, ends)
    return out


def rglru_decode(x, in_bias, conv_w, conv_b, conv_state, gates_w, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks: int,
                 out=None):
    """Decode step of a gated linear recurrent unit in one launch (one token per sequence): convolution with history
    update, block-diagonal gates, recurrence and the GELU branch."""
    n = slots.numel()
    ws = Workspace.get(x.device)
    ctr = ws._cache.get("diag_ctr")
    if ctr is None or ctr.numel() < n * blocks:
        ctr = ws._cache["diag_ctr"] = torch.zeros(max(n * blocks, 4096), dtype=torch.int32, device=x.device)
    if out is None:
        out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    ext().diag_decode(x, in_bias, conv_w, conv_b, conv_state, gates_w, gates_b, log_decay, y, y_b, state, cu_seq, slots, blocks,
                      ctr, out)
    return out


def gated_rmsnorm(o, z, w, eps, act="silu", out=None):
    C = ext()
    T, Hv, DV = o.shape
    if out is None:
        out = torch.empty_like(o)
    C.gated_rmsnorm(o, z, w, eps, Hv, DV, 0 if act == "silu" else 1, out)
    return out


def embed(ids, table, out=None):
    C = ext()
    if out is None:
        out = torch.empty(ids.numel(), table.shape[1], dtype=torch.bfloat16, device=table.device)
    C.embed(ids, table, out)
    return out
