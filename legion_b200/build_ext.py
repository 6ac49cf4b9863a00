"""In-tree build of the sm_100a extension ``legion_b200/_C.so``.

Kernel sources (``csrc/*.cu``) are compiled by nvcc for ``sm_100a`` only and carry no torch headers,
so they build in seconds; the two binding files are compiled by the host compiler against torch.
Objects are cached under ``legion_b200/csrc/build`` by source hash, so a rebuild only recompiles
what changed.  Run ``python -m legion_b200.build_ext`` (add ``-v`` for ptxas resource usage).
"""
from __future__ import annotations

import hashlib
import json
import os
import subprocess
import sys
import sysconfig
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
BUILD = CSRC / "build"
TARGET = ROOT / "_C.so"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a", "-lineinfo", "-O3", "-std=c++17", "--use_fast_math",
    "-Xcompiler", "-fPIC", "--expt-relaxed-constexpr",
]
# sources whose arithmetic serves fp32 models too: exact division, square root and exponentials, no flush to zero
PRECISE = {"hyper", "sgemm", "attn_general", "linear_scan", "resid_step", "latent_attn", "diag_scan", "logits", "conv_any",
           "channel_delta", "channel_delta_mma", "qkv_conv", "depth_step", "forget_scan"}


def _cu_flags(src: Path, verbose: bool) -> list[str]:
    flags = [f for f in NVCC_FLAGS if f != "--use_fast_math"] if src.stem in PRECISE else list(NVCC_FLAGS)
    return flags + (["-Xptxas", "-v"] if verbose else [])


def _nvcc() -> str:
    cuda_home = os.environ.get("CUDA_HOME", "/usr/local/cuda")
    cand = Path(cuda_home) / "bin" / "nvcc"
    return str(cand) if cand.exists() else "nvcc"


def _hash(path: Path, extra: str) -> str:
    h = hashlib.sha256(extra.encode())
    h.update(path.read_bytes())
    for hdr in sorted(list(CSRC.glob("*.h")) + list(CSRC.glob("*.cuh"))):
        h.update(hdr.read_bytes())
    return h.hexdigest()[:16]


def _run(cmd: list[str]) -> str:
    p = subprocess.run(cmd, capture_output=True, text=True)
    if p.returncode != 0:
        raise RuntimeError("command failed: " + " ".join(cmd) + "\n" + p.stdout + p.stderr)
    return p.stdout + p.stderr


# A checkout that has not been built compiles only the kernels of the model it is asked to run (bf16 / fp32 on one GPU):
# those every model launches, and those of its layer kinds. The binding files name all kernels; the subset is linked and
# loaded with lazy binding, so the absent ones do not matter until something calls them.
CORE_TARGET = ROOT / "_C_core.so"
CORE = {"gemm_sm100", "sgemm", "elementwise", "sampling", "spec", "tmap", "logits", "bindings", "bindings_layers"}
_ATTN = {"attn_prefill_sm100", "attn_decode_sm100", "attn_decode", "attn_general"}
_SCAN = {"linear_scan", "linear_scan_sm100", "conv1d", "conv_any"}
KIND_KERNELS = {
    "attn": _ATTN, "lightning": _SCAN, "ssd": _SCAN, "hgrn2": {"forget_scan", "forget_scan_sm100"},
    "latent": {"attn_mla_sm100", "latent_attn", "attn_prefill_sm100", "attn_decode", "attn_general"},
    "rglru": {"diag_scan", "conv1d", "conv_any"},
    "channel_delta": {"channel_delta", "channel_delta_mma"},
}


def kernels_of(cfg) -> set:
    """Source files (without suffix) a ``ModelConfig`` needs beside ``CORE``."""
    if cfg.layers is None:
        return _ATTN | {"moe", "attn_mla_sm100"}
    parts = [m for x in cfg.layers for m in ((x.mixer.left, x.mixer.right) if x.mixer.kind == "parallel" else (x.mixer,))]
    need = set().union(*(KIND_KERNELS[m.kind] for m in parts)) | {"resid_step" if cfg.sandwich_norm else "hyper"}
    if cfg.parallel_sublayers:
        need |= {"depth_step"}
    if any(a is not None and not a.direct() for a in map(cfg.attn_spec, range(cfg.n_layer))):
        need |= {"qkv_conv"}
    return need | {"moe"} if cfg.n_expert else need


def build_core(cfg, verbose: bool = False) -> Path:
    """The kernels of ``cfg``, beside those of models built before, as ``legion_b200/_C_core.so``. ``ops.sm100.ext`` takes
    it when ``_C.so`` is absent."""
    stamp = BUILD / "core.json"
    have = set(json.loads(stamp.read_text())) if stamp.exists() else set()
    need = have | kernels_of(cfg)
    out = build(verbose, core=CORE | need, force_link=need != have)
    stamp.write_text(json.dumps(sorted(need)))
    return out


def build(verbose: bool = False, force: bool = False, core: set = frozenset(), force_link: bool = False) -> Path:
    import torch
    from torch.utils import cpp_extension

    BUILD.mkdir(parents=True, exist_ok=True)
    cu_files = [f for f in sorted(CSRC.glob("*.cu")) if not core or f.stem in core]
    cpp_files = [f for f in sorted(CSRC.glob("*.cpp")) if not core or f.stem in core]
    target, module = (CORE_TARGET, "_C_core") if core else (TARGET, "_C")
    inc = [f"-I{p}" for p in cpp_extension.include_paths()] + [f"-I{sysconfig.get_paths()['include']}"]
    cuda_home = os.environ.get("CUDA_HOME", "/usr/local/cuda")
    inc.append(f"-I{cuda_home}/include")
    abi = int(torch._C._GLIBCXX_USE_CXX11_ABI)
    cxx_flags = ["-O2", "-std=c++17", "-fPIC", f"-D_GLIBCXX_USE_CXX11_ABI={abi}", f"-DTORCH_EXTENSION_NAME={module}",
                 "-DTORCH_API_INCLUDE_EXTENSION_H", "-w"] + (["-DLB_CORE"] if core else [])

    jobs = []
    objs = []
    for src in cu_files:
        flags = _cu_flags(src, verbose)
        obj = BUILD / f"{src.stem}.{_hash(src, ' '.join(flags))}.o"
        objs.append(obj)
        if force or not obj.exists():
            jobs.append(([_nvcc(), *flags, "-c", str(src), "-o", str(obj)], src))
    for src in cpp_files:
        obj = BUILD / f"{src.stem}.{_hash(src, ' '.join(cxx_flags) + torch.__version__)}.o"
        objs.append(obj)
        if force or not obj.exists():
            jobs.append((["g++", *cxx_flags, *inc, "-c", str(src), "-o", str(obj)], src))

    def work(job):
        cmd, src = job
        out = _run(cmd)
        if verbose and out.strip():
            print(f"--- {src.name}\n{out}")
        return src.name

    if jobs:
        with ThreadPoolExecutor(max_workers=min(8, len(jobs))) as ex:
            for name in ex.map(work, jobs):
                print(f"[build_ext] compiled {name}", file=sys.stderr)
    # drop stale objects of these sources
    keep = {o.name for o in objs} | {o.name for o in BUILD.glob("bindings*.o") if core}
    stems = {f.stem for f in cu_files + cpp_files}
    for o in BUILD.glob("*.o"):
        if o.name not in keep and (not core or o.name.split(".")[0] in stems):
            o.unlink()

    newest = max(o.stat().st_mtime for o in objs)
    if force or force_link or jobs or not target.exists() or target.stat().st_mtime < newest:
        torch_lib = Path(torch.__file__).parent / "lib"
        link = ["g++", "-shared", "-o", str(target), *map(str, objs), f"-L{torch_lib}", f"-L{cuda_home}/lib64",
                "-lc10", "-lc10_cuda", "-ltorch_cpu", "-ltorch_cuda", "-ltorch", "-ltorch_python", "-lcudart",
                f"-Wl,-rpath,{torch_lib}", f"-Wl,-rpath,{cuda_home}/lib64"] + (["-Wl,-z,lazy"] if core else [])
        _run(link)
        print(f"[build_ext] linked {target}", file=sys.stderr)
    return target


HOST_SRC = ROOT / "csrc_host"
HOST_TARGET = ROOT / "_host.so"


def build_host(force: bool = False) -> Path:
    """The native host runtime ``legion_b200/_host.so`` (block pool, radix cache, step packing): plain C++17 with
    pybind11, no CUDA and no torch, so it also loads in processes that never touch a GPU."""
    import pybind11
    srcs = sorted(HOST_SRC.glob("*.cpp"))
    h = hashlib.sha256()
    for s in srcs:
        h.update(s.read_bytes())
    stamp = HOST_SRC / "build" / f"host.{h.hexdigest()[:16]}.stamp"
    if not force and HOST_TARGET.exists() and stamp.exists():
        return HOST_TARGET
    stamp.parent.mkdir(parents=True, exist_ok=True)
    for old in stamp.parent.glob("host.*.stamp"):
        old.unlink()
    cmd = ["g++", "-O2", "-std=c++17", "-fPIC", "-shared", "-fvisibility=hidden", "-w",
           f"-I{pybind11.get_include()}", f"-I{sysconfig.get_paths()['include']}",
           *map(str, srcs), "-o", str(HOST_TARGET)]
    _run(cmd)
    stamp.write_text("ok")
    print(f"[build_ext] linked {HOST_TARGET}", file=sys.stderr)
    return HOST_TARGET


if __name__ == "__main__":
    build(verbose="-v" in sys.argv, force="-f" in sys.argv)
    build_host(force="-f" in sys.argv)
