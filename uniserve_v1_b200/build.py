"""Ahead-of-time build of the native libraries, in tree.

Two shared objects are produced under ``uniserve_v1_b200/_lib``:

* ``libus_kernels.so``  every ``csrc/*.cu`` compiled for sm_100a only
  (``-gencode arch=compute_100a,code=sm_100a``), plain C entry points;
* ``libus_host.so``     every ``csrc/host/*.cpp`` (block manager, batch column
  assembly, media writers): host C++ with plain C entry points.

There is no run-time kernel compilation and no Build Server process: the
reference compiles kernel packages at first start
(crates/build-server, reference project path); here the libraries are built once
and loaded with ctypes.

A *group* is the subset of sources one family needs (``GROUPS``): ``build(group=...)`` compiles
and links only those, into libraries of its own (``libus_kernels-<group>.so``), from the same
object files, so a tool that serves one model in a fresh checkout does not wait for the rest.

Usage: ``python -m uniserve_v1_b200.build [--force] [--verbose] [--group NAME]``
"""
from __future__ import annotations

import hashlib
import json
import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor
from pathlib import Path

ROOT = Path(__file__).resolve().parent
CSRC = ROOT / "csrc"
LIB = ROOT / "_lib"
OBJ = LIB / "obj"

NVCC_FLAGS = [
    "-gencode", "arch=compute_100a,code=sm_100a",
    "-lineinfo", "-O3", "-std=c++17",
    "-Xcompiler", "-fPIC,-fvisibility=hidden",
    "--expt-relaxed-constexpr",
    "-Xptxas", "-v",
]
# Sources of the families that can be built alone: (csrc/**.cu, csrc/host/*.cpp).
GROUPS = {
    "nepevik": (("runtime.cu", "gemm_tc05.cu", "linear_decode.cu", "gemm_f32.cu", "moe_route.cu",
                 "misc.cu", "sampler.cu", "row_ops.cu", "vector_delta.cu", "head_mix_attn.cu"),
                ("block_manager.cpp",)),
    "zonopel": (("runtime.cu", "gemm_tc05.cu", "linear_decode.cu", "gemm_f32.cu", "misc.cu", "sampler.cu",
                 "stream_rows.cu", "state_space.cu", "state_space_chunk.cu", "latent_attn.cu", "latent_decode.cu",
                 "latent_flash_tc05.cu"),
                ("block_manager.cpp",)),
    "tadinex": (("runtime.cu", "gemm_tc05.cu", "linear_decode.cu", "gemm_f32.cu", "moe_route.cu", "misc.cu",
                 "sampler.cu", "stream_rows.cu", "vector_delta.cu", "head_delta.cu", "state_space.cu",
                 "state_space_chunk.cu", "window_attn.cu", "latent_flash_tc05.cu", "attn_decode.cu", "attn_decode_tc05.cu"),
                ("block_manager.cpp",)),
    "nopuzen": (("runtime.cu", "gemm_tc05.cu", "linear_decode.cu", "gemm_f32.cu", "moe_route.cu", "misc.cu",
                 "sampler.cu", "stream_rows.cu", "latent_attn.cu", "latent_decode.cu", "latent_flash_tc05.cu",
                 "window_attn.cu", "sigmoid_decode.cu"),
                ("block_manager.cpp",)),
}
CXX_FLAGS = ["-O3", "-std=c++17", "-fPIC", "-fvisibility=hidden", "-pthread", "-Wall"]


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and Path(cand).exists():
            return cand
    raise RuntimeError("nvcc not found; set NVCC")


def _digest(path: Path, flags: list[str]) -> str:
    h = hashlib.sha256()
    h.update(" ".join(flags).encode())
    h.update(path.read_bytes())
    for inc in sorted((CSRC / "include").glob("*")):
        h.update(inc.read_bytes())
    return h.hexdigest()


def _compile_one(src: Path, flags: list[str], compiler: str, stamp: dict, force: bool,
                 verbose: bool) -> tuple[Path, bool, str]:
    obj = OBJ / (src.relative_to(CSRC).as_posix().replace("/", "__") + ".o")
    dig = _digest(src, flags)
    if not force and obj.exists() and stamp.get(str(obj.name)) == dig:
        return obj, False, ""
    cmd = [compiler, *flags, "-I", str(CSRC), "-c", str(src), "-o", str(obj)]
    proc = subprocess.run(cmd, capture_output=True, text=True)
    log = proc.stdout + proc.stderr
    if proc.returncode != 0:
        raise RuntimeError(f"compile failed: {' '.join(cmd)}\n{log}")
    stamp[str(obj.name)] = dig
    if verbose:
        print(log)
    return obj, True, log


def library_paths(group: str | None = None) -> tuple[Path, Path]:
    """(kernel library, host library) of the whole package or of one group."""
    tail = f"-{group}" if group else ""
    return LIB / f"libus_kernels{tail}.so", LIB / f"libus_host{tail}.so"


def _sources(group: str | None) -> tuple[list, list]:
    if group is None:
        return (sorted(CSRC.glob("*.cu")) + sorted((CSRC / "fused").glob("*.cu")),
                sorted((CSRC / "host").glob("*.cpp")))
    cu, cpp = GROUPS[group]
    return [CSRC / n for n in cu], [CSRC / "host" / n for n in cpp]


def _link(cmd: list, out: Path, objs: list, stamp: dict, force: bool) -> None:
    """Links ``objs`` into ``out`` unless it was linked from the same object digests."""
    dig = hashlib.sha256("".join(stamp[o.name] for o in objs).encode()).hexdigest()
    if not force and out.exists() and stamp.get(out.name) == dig:
        return
    tmp = out.with_suffix(f".so.tmp{os.getpid()}")       # linked aside, then moved into place at once
    proc = subprocess.run([*cmd, "-o", str(tmp), *[str(o) for o in objs]], capture_output=True,
                          text=True)
    if proc.returncode != 0:
        raise RuntimeError(f"link failed: {proc.stdout}{proc.stderr}")
    os.replace(tmp, out)
    stamp[out.name] = dig


def build(force: bool = False, verbose: bool = False, group: str | None = None) -> dict:
    """Compile what changed and link both libraries (of the package, or of one ``group``);
    returns the paths."""
    OBJ.mkdir(parents=True, exist_ok=True)
    stamp_path = OBJ / "stamp.json"
    stamp = json.loads(stamp_path.read_text()) if stamp_path.exists() else {}
    cu, cpp = _sources(group)
    nvcc = _nvcc()
    logs = {}
    with ThreadPoolExecutor(max_workers=max(1, (os.cpu_count() or 4))) as pool:
        cu_jobs = [pool.submit(_compile_one, s, NVCC_FLAGS, nvcc, stamp, force, verbose) for s in cu]
        cpp_jobs = [pool.submit(_compile_one, s, CXX_FLAGS, "g++", stamp, force, verbose)
                    for s in cpp]
        cu_res = [j.result() for j in cu_jobs]
        cpp_res = [j.result() for j in cpp_jobs]
    for (obj, _, log), src in zip(cu_res, cu):
        logs[src.name] = log
    kern, host = library_paths(group)
    _link([nvcc, "-shared", "-gencode", "arch=compute_100a,code=sm_100a", "-lcudart"], kern,
          [o for o, _, _ in cu_res], stamp, force)
    _link(["g++", "-shared", "-pthread"], host, [o for o, _, _ in cpp_res], stamp, force)
    stamp_path.write_text(json.dumps(stamp, indent=0))
    return {"kernels": kern, "host": host, "logs": logs}


def main(argv: list[str]) -> int:
    group = argv[argv.index("--group") + 1] if "--group" in argv else None
    res = build(force="--force" in argv, verbose="--verbose" in argv, group=group)
    print("built:", res["kernels"], res["host"])
    return 0


if __name__ == "__main__":
    sys.exit(main(sys.argv[1:]))
